"""Dibesun on the GPU against the plain implementation (tests/plain_dibesun.py, float64, whole sequences): each mechanism
alone (the norm in parts with and without a delta, the norm over whole query and key rows, linear attention by the scan,
in chunks and token by token, the gate behind it, SiLU on a range of columns, the router's bias, one layer against plain
models with one constant or one rule changed), whole prompts, prompts then token-by-token decoding across page and chunk
borders, portions down to two tokens, batches of unequal requests against each alone, slots and pages that are used again,
keys that stand out just inside and just outside a chunk (in prompts and decoded), the first tokens of a sequence, long
decoding, and greedy generation through `Engine.generate`, the command line and the trace runner. Weights and
configurations are the tests' own (tests/dibesun_configs.py)."""
import copy
import json
import types

import numpy as np
import pytest
import torch

import dibesun_configs as configs
import plain_dibesun

pytestmark = pytest.mark.gpu

# Bounds on a request's logits: the largest difference relative to the largest logit, and the root mean square of the
# differences relative to that of the logits.
BOUND = {"float32": 1e-5, "bfloat16": 0.04}
LARGEST = {"float32": 4e-5, "bfloat16": 0.2}
GREEDY = {"float32": 2e-5, "bfloat16": 0.04}      # two logits closer than this (relative to the largest) may swap


# In bfloat16 a router's choice between experts whose logits lie closer together than the rounding of its input may fall
# the other way. Where a test compares whole models, the plain model takes the engine's choice at such a token, but only if
# moving the logits by this much towards it makes it the plain model's own choice.
CLOSE_CALL = 0.12
_routes = []                # what the router chose, call by call


@pytest.fixture(autouse=True)
def recorded_routes(monkeypatch):
    from kidi_b200.kernels import routed
    route = routed.route

    def recorded(*args, **kwargs):
        chosen, weight = route(*args, **kwargs)
        if not torch.cuda.is_current_stream_capturing():
            _routes.append(chosen)
        return chosen, weight

    monkeypatch.setattr(routed, "route", recorded)


def make(config, dtype, seed=1, max_tokens=2048, tensors=None, **weights):
    """(engine, tensors). `engine.choices[slot]`: for every routed layer the experts chosen for the tokens of the sequence
    that holds (or last held) the slot, [tokens, top]."""
    from kidi_b200 import Engine
    tensors = tensors or configs.tensors(config, seed, **weights)
    engine = Engine.from_config(config, tensors=tensors, dtype=dtype, max_tokens=max_tokens)
    engine.choices, step = {}, engine.step

    def recording_step(batch):
        fresh = [engine.cache.length(slot) == 0 for slot in batch.slots]
        before = len(_routes)
        logits = step(batch)
        made, at = [chosen.cpu() for chosen in _routes[before:]], 0
        for slot, tokens, new in zip(batch.slots, batch.tokens, fresh):
            rows = [chosen[at:at + len(tokens)] for chosen in made]
            engine.choices[slot] = rows if new else [torch.cat(pair) for pair in zip(engine.choices[slot], rows)]
            at += len(tokens)
        return logits

    engine.step = recording_step
    return engine, tensors


def prompt(config, length, seed):
    return np.random.default_rng(seed).integers(0, config["vocab"], size=length).tolist()


def plain(config, tensors, tokens, choices=None):
    return plain_dibesun.forward(config, tensors, tokens, dtype=torch.float64, choices=choices, margin=CLOSE_CALL)


def follow(engine, slot, dtype, config, tensors, tokens, want):
    """The plain model's logits; in bfloat16 with the engine's choices where the plain model's own are close calls."""
    if dtype == "float32" or not engine.choices[slot]:
        return want
    return plain(config, tensors, tokens, engine.choices[slot])


def run(engine, slot, tokens, want=None):
    from kidi_b200 import StepBatch
    want = list(range(len(tokens))) if want is None else want
    return engine.step(StepBatch([slot], [list(tokens)], [want])).double().cpu()


def close(got, want, dtype, record=None, what="", slack=1.0):
    assert torch.isfinite(got).all(), what
    scale, level = float(want.abs().max()), float(want.pow(2).mean().sqrt())
    worst = float((got - want).abs().max()) / scale
    mean = float((got - want).pow(2).mean().sqrt()) / level
    if record is not None:
        record(f"largest and mean relative difference {what}".strip(), (worst, mean))
    assert worst < slack * LARGEST[dtype] and mean < slack * BOUND[dtype], (what, worst, mean, scale)


def nearer(got, want, others, what, rows=slice(None)):
    """`got` lies nearer to `want` than to any of `others` (plain models with one thing changed)."""
    right = float((got[rows] - want[rows]).pow(2).mean().sqrt())
    for index, other in enumerate(others):
        assert right < 0.5 * float((got[rows] - other[rows]).pow(2).mean().sqrt()), (what, index)


def in_steps(engine, tokens, sizes):
    slot = engine.acquire()
    rows, at = [], 0
    for size in sizes:
        rows.append(run(engine, slot, tokens[at:at + size]))
        at += size
    assert at == len(tokens)
    engine.release(slot)
    return torch.cat(rows)


def decoded(engine, tokens, head):
    return in_steps(engine, tokens, [head] + [1] * (len(tokens) - head))


def changed(config, path, value):
    other = copy.deepcopy(config)
    node = other
    for key in path[:-1]:
        node = node[key]
    if value is None:
        del node[path[-1]]
    else:
        node[path[-1]] = value
    return other


def step_tables(lengths, starts, slots):
    """The device tables of a step that brings `lengths[b]` tokens to sequences that hold `starts[b]`."""
    row_seq, row_pos, row0, cursor = [], [], [], 0
    for index, (count, start) in enumerate(zip(lengths, starts)):
        row0.append(cursor)
        row_seq += [index] * count
        row_pos += list(range(start, start + count))
        cursor += count
    as_int = lambda values: torch.tensor(values, dtype=torch.int32).cuda()
    return types.SimpleNamespace(row_seq=as_int(row_seq), row_pos=as_int(row_pos), seq_slot=as_int(slots),
                                 seq_start=as_int(starts), seq_row0=as_int(row0), seq_len=as_int(lengths))


# ------------------------------------------------------------------ the kernels alone
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hidden,groups,delta_groups", [(48, 3, 1), (50, 1, 5), (1024, 8, 2), (1024, 16, 1), (2048, 1, 4),
                                                        (3072, 24, 3), (272, 17, 1), (4096, 32, 8), (8192, 2, 64)])
def test_the_norm_in_parts(dtype, hidden, groups, delta_groups):
    """stream += norm(delta) and the norm of the sum, or a copy of it; at picked rows the stream stays as it is."""
    from kidi_b200.kernels import ops
    generator = torch.Generator().manual_seed(hidden + groups)
    loose = dict(atol=2e-5, rtol=1e-5) if dtype == torch.float32 else dict(atol=2e-2, rtol=1e-2)
    rows = 5
    stream = torch.randn(rows, hidden, generator=generator) * 3
    delta = (torch.randn(rows, hidden, generator=generator) * torch.rand(rows, hidden, generator=generator) * 4).to(dtype)
    weight, outer = (torch.randn(hidden, generator=generator) * 0.3 + 1 for _ in range(2))
    total = stream.double() + plain_dibesun.grouped_rms(delta.double(), outer, 1e-3, delta_groups)
    normed = plain_dibesun.grouped_rms(total, weight, 1e-5, groups)
    args = dict(delta_weight=outer.cuda(), delta_groups=delta_groups, delta_eps=1e-3)
    index = torch.tensor([4, 0, 4], dtype=torch.int32).cuda()
    held = stream.cuda()
    got = ops.add_parts_norm(held, delta.cuda(), dtype, weight=weight.cuda(), groups=groups, eps=1e-5, row_index=index, **args)
    assert torch.allclose(got.double().cpu(), normed[[4, 0, 4]], **loose) and torch.equal(held.cpu(), stream)
    got = ops.add_parts_norm(held, delta.cuda(), dtype, weight=weight.cuda(), groups=groups, eps=1e-5, **args)
    assert torch.allclose(got.double().cpu(), normed, **loose)
    assert torch.allclose(held.double().cpu(), total, atol=2e-5, rtol=1e-6)
    held = stream.cuda()
    got = ops.add_parts_norm(held, delta.cuda(), dtype, **args)                       # a copy of the stream
    assert torch.equal(got, held.to(dtype)) and torch.allclose(held.double().cpu(), total, atol=2e-5, rtol=1e-6)
    held = stream.cuda()
    got = ops.add_parts_norm(held, delta.cuda(), dtype)                               # a delta that passes no norm
    assert torch.allclose(held.double().cpu(), stream.double() + delta.double(), atol=1e-5) and torch.equal(got, held.to(dtype))
    assert ops.add_parts_norm(held, None, None) is None


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,ring", [(4, 2, 16, 16, 0), (3, 1, 10, 6, 0), (40, 8, 128, 128, 0),
                                                          (6, 3, 24, 40, 2), (72, 36, 64, 64, 1)])
def test_the_norm_over_whole_rows_and_its_cache_write(dtype, heads, kv_heads, dim, vdim, ring):
    """Queries and keys of a row divided by one root mean square each, keys and values in the cache's pages (also where
    they lie beyond a ring's reach: not written), a padding row left alone, columns behind the values left alone."""
    from kidi_b200.kernels import ops
    generator = torch.Generator().manual_seed(heads)
    lengths, starts, slots = (70, 3), (60, 0), (2, 0)
    rows, width = sum(lengths), (heads + kv_heads) * dim + kv_heads * vdim
    pad = 8 + (-width % 8)
    qkv = torch.randn(rows, width + pad, generator=generator).to(dtype)
    q_norm, k_norm = (torch.randn(n, generator=generator) * 0.3 + 1 for n in (heads * dim, kv_heads * dim))
    tables = step_tables(lengths, starts, slots)
    tables.row_seq[72] = -1
    pages_per = ring or 3
    keys = torch.zeros(3 * pages_per, kv_heads, 64, dim, dtype=dtype).cuda()
    values = torch.zeros(3 * pages_per, kv_heads, 64, vdim, dtype=dtype).cuda()
    table = torch.randperm(3 * pages_per, generator=generator).reshape(3, pages_per).int()
    view = types.SimpleNamespace(keys=keys, values=values, table=table.cuda(), page_size=64, ring_pages=ring)
    held = qkv.cuda()
    ops.wide_norm_store(held, heads=heads, kv_heads=kv_heads, head_dim=dim, value_dim=vdim, q_norm=q_norm.cuda(),
                        k_norm=k_norm.cuda(), eps=1e-5, tables=tables, kv_view=view, store=True)
    split = heads * dim, (heads + kv_heads) * dim
    want = qkv.double().clone()
    want[:, :split[0]] = plain_dibesun.grouped_rms(want[:, :split[0]], q_norm, 1e-5)
    want[:, split[0]:split[1]] = plain_dibesun.grouped_rms(want[:, split[0]:split[1]], k_norm, 1e-5)
    want[72] = qkv[72].double()
    got = held.double().cpu()
    assert torch.allclose(got, want, atol=1e-5 if dtype == torch.float32 else 3e-2)
    assert torch.equal(held[:, split[1]:].cpu(), qkv[:, split[1]:])
    at = 0
    for b, (count, start) in enumerate(zip(lengths, starts)):
        for t in range(count):
            row, position = at + t, start + t
            if ring and position < start + count - 64 * ring:
                continue                                        # a later token of the step took its place
            page = table[slots[b], (position // 64) % pages_per]
            stored = keys[page, :, position % 64].cpu(), values[page, :, position % 64].cpu()
            if row == 72:
                assert not stored[0].any() and not stored[1].any()
                continue
            assert torch.equal(stored[0].reshape(-1), held[row, split[0]:split[1]].cpu())
            assert torch.equal(stored[1].reshape(-1), held[row, split[1]:width].cpu())
        at += count


@pytest.mark.parametrize("form", ["scan", "chunks", "bits"])
@pytest.mark.parametrize("heads,dim,vdim", [(3, 16, 48), (2, 32, 64), (5, 48, 16), (2, 128, 128)])
def test_linear_attention_in_portions(heads, dim, vdim, form, monkeypatch):
    """The scan, the chunked tensor-core form and the one-token kernel against the loop over each sequence (decays of 0
    and 1 among them), with states that are carried in and slots in any order: portions that are whole chunks, a token
    more and less than one, single tokens; the scan's results do not depend on the cut."""
    from kidi_b200.kernels import linear_attention as kernels
    from kidi_b200.kernels import ops
    dtype = torch.float32 if form == "bits" else torch.bfloat16
    monkeypatch.setattr(kernels, "MIN_CHUNKED_TOKENS", 2 if form == "chunks" else 0)
    generator = torch.Generator().manual_seed(dim)
    lengths, slots = (200, 1, 131), (2, 0, 4)
    total, width = sum(lengths), heads * (2 * dim + vdim)
    packed = torch.randn(total, width + 8, generator=generator).to(dtype)
    decay = torch.tensor(([0.0, 1.0] + [0.9 + 0.02 * h for h in range(heads)])[:heads])
    start = torch.randn(6, heads, dim, vdim, generator=generator)
    parts = lambda x: (x[:, :heads * dim], x[:, heads * dim:2 * heads * dim], x[:, 2 * heads * dim:width])
    want, states, at = [], [], 0
    for b, count in enumerate(lengths):
        q, k, v = (x[at:at + count].double() for x in parts(packed))
        S = start[slots[b]].double().clone()
        want.append(plain_dibesun.fixed_decay_recurrence(q.reshape(count, heads, dim), k.reshape(count, heads, dim),
                                                         v.reshape(count, heads, vdim), decay.tolist(), S).reshape(count, -1))
        states.append(S)
        at += count
    found = []
    for cuts in ((200, 131), (64, 65), (63, 128), (100, 7), (199, 130)):
        state = start.clone().cuda()
        pieces, done = [[] for _ in lengths], [0] * len(lengths)
        with ops.record_launches() as names:
            while any(d < n for d, n in zip(done, lengths)):
                live = [b for b, n in enumerate(lengths) if done[b] < n]
                sizes = [min(lengths[b] - done[b], cuts[0] if b == 0 else cuts[1]) for b in live]
                rows = torch.cat([torch.arange(sum(lengths[:b]) + done[b], sum(lengths[:b]) + done[b] + n)
                                  for b, n in zip(live, sizes)])
                q, k, v = parts(packed[rows].cuda())
                out = kernels.linear_attention(q, k, v, decay.cuda(), state, heads=heads, dim=dim, vdim=vdim,
                                               tables=step_tables(sizes, [done[b] for b in live], [slots[b] for b in live]),
                                               seqs=len(live), one_token=max(sizes) == 1, longest=max(sizes)).cpu()
                at = 0
                for b, n in zip(live, sizes):
                    pieces[b].append(out[at:at + n])
                    at += n
                    done[b] += n
        assert ("linear_attention[chunks]" if form == "chunks" else "scalar_recurrence") in names
        if cuts[0] == 199:
            assert "linear_attention[one token]" in names
        found.append([torch.cat(p) for p in pieces])
        for b in range(len(lengths)):
            scale = float(want[b].abs().max())
            assert float((found[-1][b].double() - want[b]).abs().max()) < 4e-6 * scale, (cuts, b)
            scale = float(states[b].abs().max())
            assert float((state[slots[b]].double().cpu() - states[b]).abs().max()) < 4e-6 * scale, (cuts, b)
        untouched = [slot for slot in range(6) if slot not in slots]
        assert torch.equal(state[untouched].cpu(), start[untouched])
    if form == "bits":
        assert all(torch.equal(a, b) for cut in found[1:4] for a, b in zip(cut, found[0]))


def test_the_chunked_form_takes_heads_in_groups(monkeypatch):
    """With little scratch memory the heads of a step run in several launches: the same bits."""
    from kidi_b200.kernels import linear_attention as kernels
    from kidi_b200.kernels import ops
    generator = torch.Generator().manual_seed(8)
    heads, dim, vdim, rows = 5, 32, 64, 150
    q, k, v = (torch.randn(rows, heads * n, generator=generator).bfloat16().cuda() for n in (dim, dim, vdim))
    decay = torch.rand(heads, generator=generator).cuda()
    results = []
    for floats in (1 << 30, 1):
        monkeypatch.setattr(kernels, "SCRATCH_FLOATS", floats)
        state = torch.zeros(2, heads, dim, vdim).cuda()
        with ops.record_launches() as names:
            out = kernels.linear_attention(q, k, v, decay, state, heads=heads, dim=dim, vdim=vdim,
                                           tables=step_tables([rows], [0], [1]), seqs=1, one_token=False, longest=rows)
        results.append((out.cpu(), state.cpu()))
        assert names.count("linear_attention[chunks]") == (1 if floats > 1 else heads)
    assert torch.equal(results[0][0], results[1][0]) and torch.equal(results[0][1], results[1][1])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_one_token_steps_of_the_recurrence(dtype):
    """The one-token kernel at widths with and without 16-byte pieces, more state rows than one pass takes, and a padding
    sequence whose slot stays as it is."""
    from kidi_b200.kernels import linear_attention as kernels
    for heads, dim, vdim in ((2, 7, 5), (3, 256, 36), (1, 130, 33), (4, 16, 128)):
        generator = torch.Generator().manual_seed(dim)
        q, k, v = (torch.randn(3, heads * n, generator=generator).to(dtype) for n in (dim, dim, vdim))
        decay = torch.rand(heads, generator=generator)
        start = torch.randn(4, heads, dim, vdim, generator=generator)
        state, tables = start.clone().cuda(), step_tables([1, 1, 1], [9, 0, 0], [2, 3, 0])
        tables.row_seq[1] = -1
        out = kernels.linear_attention(q.cuda(), k.cuda(), v.cuda(), decay.cuda(), state, heads=heads, dim=dim, vdim=vdim,
                                       tables=tables, seqs=3, one_token=True, longest=1).double().cpu()
        for b, slot in ((0, 2), (2, 0)):
            S = start[slot].double()
            want = plain_dibesun.fixed_decay_recurrence(q[b:b + 1].double().reshape(1, heads, dim), k[b:b + 1].double().reshape(1, heads, dim),
                                                        v[b:b + 1].double().reshape(1, heads, vdim), decay.tolist(), S)
            assert torch.allclose(out[b], want.reshape(-1), atol=2e-5 * dim ** 0.5, rtol=1e-5)
            assert torch.allclose(state[slot].double().cpu(), S, atol=1e-5)
        assert torch.equal(state[[1, 3]].cpu(), start[[1, 3]])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_gate_behind_the_recurrence_and_silu_on_columns(dtype):
    from kidi_b200.kernels import linear_attention as kernels
    from kidi_b200.kernels import skinny
    loose = dict(atol=2e-5, rtol=1e-5) if dtype == torch.float32 else dict(atol=2e-2, rtol=1e-2)
    generator = torch.Generator().manual_seed(3)
    for rows, width in ((3, 45), (2, 64), (1, 4096), (2, 6000)):
        read = torch.randn(rows, width, generator=generator) * 5
        weight = torch.randn(width, generator=generator) * 0.3 + 1
        gate = (torch.randn(rows, width + 8, generator=generator) * 2).to(dtype)
        out = torch.zeros(rows, width + 16, dtype=dtype).cuda()
        kernels.normed_gate(read.cuda(), weight.cuda(), gate.cuda()[:, 8:], 1e-5, -0.6, out[:, 8:8 + width])
        want = -0.6 * plain_dibesun.grouped_rms(read.double(), weight, 1e-5) * torch.sigmoid(gate[:, 8:].double())
        assert torch.allclose(out[:, 8:8 + width].double().cpu(), want, **loose)
        assert not out[:, :8].any() and not out[:, 8 + width:].any()
    for width, begin, end in ((48, 8, 40), (48, 3, 29), (21, 0, 21), (16, 5, 5)):
        x = torch.randn(4, width, generator=generator).to(dtype)
        want = x.double().clone()
        want[:, begin:end] = plain_dibesun.silu(want[:, begin:end])
        assert torch.allclose(kernels.silu_columns(x.cuda(), begin, end).double().cpu(), want, **loose)
    if dtype == torch.bfloat16:                        # the same in the weight-streaming product's epilogue
        x, weight = torch.randn(5, 72, generator=generator).bfloat16(), torch.randn(100, 72, generator=generator).bfloat16()
        want = x.double() @ weight.double().t()
        want[:, 9:90] = plain_dibesun.silu(want[:, 9:90])
        got = skinny.gemm(x.cuda(), weight.cuda(), torch.float32, silu_columns=(9, 90)).double().cpu()
        assert torch.allclose(got, want, atol=1e-3, rtol=1e-4)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_router_with_a_bias(dtype):
    """The bias counts in the choice and in the weights; renormalised without an addend the weights are the softmax over
    the chosen logits, also where the others lie far below."""
    from kidi_b200.kernels import routed
    generator = torch.Generator().manual_seed(5)
    for experts, top in ((6, 2), (16, 4), (40, 40), (3, 1)):
        x = torch.randn(9, 64, generator=generator).to(dtype)
        router = (torch.randn(experts, 64, generator=generator)).to(dtype)
        bias = torch.randn(experts, generator=generator) * 6
        z = x.double() @ router.double().t() + bias.double()
        if top <= 32:
            chosen, weight = routed.route(x.cuda(), router.cuda(), top, True, "softmax", bias=bias.cuda())
            best = torch.topk(z, top)
            assert torch.equal(chosen.cpu().long(), best.indices)
            assert torch.allclose(weight.double().cpu(), torch.softmax(best.values, -1), atol=1e-5)


# ------------------------------------------------------------------ one layer
ONE = configs.layer(configs.attention(4, 2, 16, 24, 0.4, chunk=70, softcap=3.0), configs.linear(3, 12, 20, (0.6, 0.95, 0.999)),
                    configs.routed(6, 2, 24, shared=16), left_scale=1.1, right_scale=0.6)
# what must not be confused with what: (path into the configuration, other value); None removes the key; a pair of values:
# the finer one for 32-bit, the coarser one where bfloat16 rounding would drown the finer
MIX = ("layers", 0, "mixer")
OTHERS = [(MIX + ("left", "mask", "size"), 69), (MIX + ("left", "mask", "size"), 71), (MIX + ("left", "mask"), None),
          (MIX + ("left", "softcap"), (2.8, 1.5)), (MIX + ("left", "softcap"), None), (MIX + ("left", "scale"), (0.38, 0.2)),
          (MIX + ("left_scale",), 0.8), (MIX + ("right_scale",), 0.3), (MIX + ("right", "decay"), [0.95, 0.6, 0.999]),
          (("norm", "groups"), 1), (("norm", "groups"), 6), (("embedding", "scale"), 1.5),
          (("layers", 0, "mlp", "router", "top"), 3)]


def other_rules(monkeypatch, config, tensors, tokens):
    """Plain models with one rule changed: a sliding window instead of chunks, chunks that start one position later, a
    softmax instead of sigmoids, no number added to the scores, norms of q and k head by head, a router without bias, no
    shared expert, a head that has the embedding's scale."""
    found = []

    def with_patch(name, replacement):
        with monkeypatch.context() as patch:
            patch.setattr(plain_dibesun, name, replacement)
            found.append(plain(config, tensors, tokens))

    size = config["layers"][0]["mixer"]["left"]["mask"]["size"]
    i, j = torch.arange(len(tokens))[:, None], torch.arange(len(tokens))[None, :]
    with_patch("same_chunk", lambda T, _: (j <= i) & (i - j < size))
    with_patch("same_chunk", lambda T, _: (j <= i) & ((i + 1) // size == (j + 1) // size))
    with_patch("sigmoid_weights", lambda s, seen, bias: torch.softmax((s + bias).masked_fill(~seen, float("-inf")), -1))
    left = config["layers"][0]["mixer"]["left"]
    whole = plain_dibesun.grouped_rms

    def by_head(x, weight, eps, groups=1):
        heads = {left["heads"] * left["dim"]: left["heads"], left["kv_heads"] * left["dim"]: left["kv_heads"]}
        return whole(x, weight, eps, heads.get(x.shape[-1], groups))

    with_patch("grouped_rms", by_head)
    for names in (("mix.left.pb",), ("router.b",), ("shared.down",), ("mix.right.g",)):
        without = {name: torch.zeros_like(t) if name.endswith(names) else t for name, t in tensors.items()}
        found.append(plain(config, without, tokens))
    return found


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_one_layer_alone(dtype, monkeypatch, record_property):
    """A model of one layer, whole, in portions and decoded over three pages and chunks, against the plain model and
    against plain models with one constant or rule changed: the engine's logits must lie nearer to the right one."""
    config = configs.single(ONE, groups=3)
    engine, tensors = make(config, dtype, seed=11, sharp=2.0, logits=4.0)
    tokens = prompt(config, 220, 21)
    want = plain(config, tensors, tokens)
    pick = lambda value: value[dtype == "bfloat16"] if isinstance(value, tuple) else value
    others = [plain(changed(config, path, pick(value)), tensors, tokens) for path, value in OTHERS]
    others += other_rules(monkeypatch, config, tensors, tokens)
    for what, got in (("whole", in_steps(engine, tokens, [220])),
                      ("in portions", in_steps(engine, tokens, [61, 2, 3, 64, 1, 30, 59])),
                      ("decoded", decoded(engine, tokens, 50))):
        close(got, want, dtype, record_property, what)
        nearer(got, want, others, what, rows=slice(68, 220))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("chunk,width", [(40, 16), (64, 64), (130, 64), (150, 24), (128, 48), (1, 16)])
def test_a_key_that_stands_out_at_a_chunks_edge(dtype, chunk, width, record_property):
    """Almost every weight is near zero (a large negative number on the scores) except that of a key whose token also has
    the query's direction: the same special token stands first in a chunk, last in the chunk before it, and is asked for by
    rows just behind and by the chunk's last row, in a prompt, in portions and decoded. Against plain models whose chunks
    are one position shorter or longer."""
    one = configs.layer(configs.attention(2, 1, width, width, 4.0, chunk=chunk, softcap=60.0), configs.linear(1, 8, 8),
                        left_scale=1.5, right_scale=0.25)
    config = configs.single(one, width=48, groups=1)
    tensors = configs.tensors(config, 3, logits=3.0)
    special, mark = 5, torch.zeros(48)
    mark[7] = 1.0
    table = tensors["embed"].float() * 0.7
    table[:, 7] = 0.0
    table[special] = mark * 6.0                            # the only token with anything in channel 7 (and nothing else)
    asking = 9
    table[asking, 7] = 3.0
    tensors["embed"] = table.bfloat16()
    for name in "qk":
        matrix = torch.zeros_like(tensors[f"l0.mix.left.{name}"].float()) + 0.02 * tensors[f"l0.mix.left.{name}"].float()
        matrix[::width if name == "k" else width, 7] = 1.0   # the first entry of each head reads channel 7
        tensors[f"l0.mix.left.{name}"] = matrix.bfloat16()
        tensors[f"l0.mix.left.{name}.norm"] = torch.ones_like(tensors[f"l0.mix.left.{name}.norm"])
    tensors["l0.mix.left.pb"] = torch.full_like(tensors["l0.mix.left.pb"], -12.0)
    engine, _ = make(config, dtype, tensors=tensors)
    tokens = [t if t not in (special, asking) else 11 for t in prompt(config, 3 * chunk + 20 if chunk > 1 else 70, 4)]
    edge = 2 * chunk
    asked = [edge - 1, edge, edge + 1, min(len(tokens) - 1, edge + chunk - 1)]
    wrong = [plain_model_of(config, tensors, size) for size in ([chunk - 1, chunk + 1] if chunk > 1 else [2])]
    for place in (edge - 1, edge):                         # the chunk's last position before the edge, the first behind it
        sequence = list(tokens)
        for row in asked:
            sequence[row] = asking
        sequence[place] = special
        want = plain(config, tensors, sequence)
        rows = [row for row in asked if row > place] or [place]
        others = [model(sequence) for model in wrong]
        level = 0.04 * float(want.abs().max())
        felt = [(other, [row for row in rows if float((other[row] - want[row]).abs().max()) > level]) for other in others]
        assert chunk == 1 or all(where for _, where in felt), "the edge does not show"
        for what, got in (("whole", in_steps(engine, sequence, [len(sequence)])),
                          ("portions", in_steps(engine, sequence, [edge - 1, 2, len(sequence) - edge - 1])),
                          ("decoded", decoded(engine, sequence, max(1, edge - 2)))):
            close(got, want, dtype, record_property, f"{what}, key at {place - edge}")
            for other, where in felt:
                if where:
                    nearer(got, want, [other], what, rows=where)


def plain_model_of(config, tensors, size):
    return lambda tokens: plain(changed(config, MIX + ("left", "mask", "size"), size), tensors, tokens)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("chunk", [None, 150])
def test_far_tokens_reach_the_last_rows(dtype, chunk, record_property):
    """600 tokens: the state of a slowly decaying head (and attention without chunks) carries the first forty tokens to the
    last rows; with quickly decaying heads and chunks of 150 nothing of them is left. Whole, in portions and decoded."""
    decay = (0.999, 1.0) if chunk is None else (0.3, 0.5)
    config = configs.single(configs.layer(configs.attention(2, 1, 16, 16, 0.6, chunk=chunk, softcap=30.0),
                                          configs.linear(2, 16, 16, decay)), groups=2)
    engine, tensors = make(config, dtype, seed=13, sharp=3.0)
    tokens = prompt(config, 600, 3)
    other = prompt(config, 40, 4) + tokens[40:]
    want, moved = plain(config, tensors, tokens), plain(config, tensors, other)
    shift = float((want[560:] - moved[560:]).abs().max()) / float(want.abs().max())
    record_property("what the first forty tokens move the last rows by", shift)
    assert shift > 0.02 if chunk is None else shift < 1e-12
    for sequence, expected in ((tokens, want), (other, moved)):
        close(in_steps(engine, sequence, [600])[560:], expected[560:], dtype, record_property, "whole")
        close(in_steps(engine, sequence, [333, 2, 265])[560:], expected[560:], dtype, record_property, "in portions")
        close(decoded(engine, sequence, 400)[560:], expected[560:], dtype, record_property, "decoded")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_state_starts_at_zero_in_a_used_slot(dtype):
    config = configs.single(ONE)
    engine, tensors = make(config, dtype, seed=5)
    slot = engine.acquire()
    run(engine, slot, prompt(config, 90, 1))
    engine.release(slot)
    for length in (1, 2, 3, 5, 40):
        tokens = prompt(config, length, 30 + length)
        assert engine.acquire() == slot
        got = run(engine, slot, tokens)
        engine.release(slot)
        close(got, plain(config, tensors, tokens), dtype, what=f"{length} tokens")
        close(decoded(engine, tokens, 1), plain(config, tensors, tokens), dtype, what=f"{length} tokens decoded")


# ------------------------------------------------------------------ whole models
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(configs.ALL))
def test_whole_prompts_portions_and_decoding(name, dtype, record_property):
    config = configs.ALL[name]
    engine, tensors = make(config, dtype, seed=2)
    tokens = prompt(config, 330 if name == "wide" else 210, 9)
    plainly = plain(config, tensors, tokens)
    for what, sizes in (("whole", [len(tokens)]), ("in portions", [63, 2, 64, 1, 3, len(tokens) - 133]),
                        ("two by two", [2] * 30 + [len(tokens) - 60]),
                        ("decoded past every chunk", [len(tokens) - 190] + [1] * 190)):
        got = in_steps(engine, tokens, sizes)
        (slot,) = engine.choices                              # one slot serves every run
        close(got, follow(engine, slot, dtype, config, tensors, tokens, plainly), dtype, record_property, what)
    for length in (1, 2, 3):
        few = prompt(config, length, 50 + length)
        close(in_steps(engine, few, [length]), plain(config, tensors, few), dtype, what=f"{length} tokens")
    engine.cache.check()
    assert not engine.cache.slots.held
    engine.check_device_errors()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(configs.ALL))
def test_batches_of_unequal_requests(name, dtype, record_property):
    """Requests of unequal lengths start together, are decoded together, the shorter ones leave and their slots and
    pages go to the next batch at once: every request as if it ran alone."""
    from kidi_b200 import StepBatch
    config = configs.ALL[name]
    engine, tensors = make(config, dtype, seed=4, max_tokens=1024)
    seen = set()
    for batch, sizes in enumerate([(1, 70, 131, 40), (150, 3, 66), (90, 64)]):
        requests = [prompt(config, n + 6 + 3 * i, 100 * batch + i) for i, n in enumerate(sizes)]
        want = [plain(config, tensors, r) for r in requests]
        slots = [engine.acquire() for _ in requests]
        if batch:
            assert seen & set(slots)                       # slots (and their pages) are used again
        seen |= set(slots)
        logits = engine.step(StepBatch(slots, [r[:n] for r, n in zip(requests, sizes)],
                                       [list(range(n)) for n in sizes])).double().cpu()
        got, at = [], 0
        for n in sizes:
            got.append([logits[at:at + n]])
            at += n
        done, live = list(sizes), list(range(len(requests)))
        while live:
            step = engine.step(StepBatch([slots[b] for b in live], [[requests[b][done[b]]] for b in live],
                                         [[0]] * len(live))).double().cpu()
            for row, b in enumerate(live):
                got[b].append(step[row:row + 1])
                done[b] += 1
            for b in [b for b in live if done[b] == len(requests[b])]:
                engine.release(slots[b])
            live = [b for b in live if done[b] < len(requests[b])]
        for b, expected in enumerate(want):
            expected = follow(engine, slots[b], dtype, config, tensors, requests[b], expected)
            close(torch.cat(got[b]), expected, dtype, record_property, f"batch {batch}, request {b}")
    engine.cache.check()
    assert not engine.cache.slots.held


def test_a_dozen_sequences_decode_together(record_property):
    """More rows than the weight-streaming product takes, and the wider kernels of prompts: twelve sequences."""
    from kidi_b200 import StepBatch
    config = configs.WIDE
    engine, tensors = make(config, "bfloat16", seed=4, max_tokens=4096)
    requests = [prompt(config, 20 + 17 * i, i) for i in range(12)]
    slots = [engine.acquire() for _ in requests]
    engine.step(StepBatch(slots, [r[:-2] for r in requests], [[]] * 12))
    first = engine.step(StepBatch(slots, [[r[-2]] for r in requests], None)).double().cpu()
    last = engine.step(StepBatch(slots, [[r[-1]] for r in requests], None)).double().cpu()
    want = [plain(config, tensors, r, engine.choices[slot]) for r, slot in zip(requests, slots)]
    close(torch.cat([first, last]), torch.stack([w[-2] for w in want] + [w[-1] for w in want]), "bfloat16", record_property)


def test_batches_and_portions_leave_32_bit_logits_alone():
    """In 32-bit a request's logits are the same alone, in a batch and in portions (within 4e-6 of the largest)."""
    from kidi_b200 import StepBatch
    config = configs.SMALL_A
    engine, tensors = make(config, "float32", seed=6)
    a, b = prompt(config, 150, 1), prompt(config, 77, 2)
    alone = in_steps(engine, a, [150])
    cut = in_steps(engine, a, [64, 2, 83, 1])
    slots = [engine.acquire(), engine.acquire()]
    both = engine.step(StepBatch(slots, [b, a], [[76], list(range(150))])).double().cpu()[1:]
    for slot in slots:
        engine.release(slot)
    scale = float(alone.abs().max())
    assert float((alone - cut).abs().max()) <= 4e-6 * scale and float((alone - both).abs().max()) <= 4e-6 * scale


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_prompts_and_long_decoding(dtype, record_property):
    """A prompt of more than 1,024 tokens (the tensor-memory products, many chunks of both kinds) and 300 decoded tokens."""
    config = configs.model(101, 128, 1e-5, 2, 3.0, [
        configs.layer(configs.attention(4, 2, 64, 64, 0.15, chunk=300, softcap=20.0), configs.linear(2, 64, 64, (0.9, 0.9995))),
        configs.layer(configs.attention(2, 2, 16, 16, 0.3, softcap=20.0), configs.linear(3, 16, 16), configs.dense(64))],
        positions=1600)
    engine, tensors = make(config, dtype, seed=8, max_tokens=4096)
    tokens = prompt(config, 1400, 2)
    want = plain(config, tensors, tokens)
    close(in_steps(engine, tokens, [1400]), want, dtype, record_property, "whole")
    close(decoded(engine, tokens, 1100), want, dtype, record_property, "decoded")


def test_which_kernels_run(record_property):
    """The bfloat16 engine takes the tensor-core attention kernels with sigmoid weights (tcgen05 for prompts at head widths
    64 and 128, mma.sync else, and in decoding), chunked linear attention for prompts and the one-token kernel in decoding;
    the 32-bit engine takes the general kernels and the 32-bit product only."""
    from kidi_b200.kernels import ops
    config = configs.WIDE
    engine, tensors = make(config, "bfloat16", seed=3)
    tokens = prompt(config, 300, 5)
    want = plain(config, tensors, tokens)
    slot = engine.acquire()
    with ops.record_launches() as names:
        run(engine, slot, tokens[:299], want=[])
    record_property("prompt kernels", sorted(set(names)))
    assert names.count("attention_prefill_tcgen05") == 3 and names.count("attention_prefill[mma.sync]") == 2
    assert names.count("linear_attention[chunks]") == 4 and names.count("scalar_recurrence") == 1      # heads of 24 x 40
    assert names.count("wide_norm_store") == 5 and names.count("normed_gate") == 5 and "attention" not in names
    with ops.record_launches() as names:
        last = run(engine, slot, tokens[299:])
    record_property("decode kernels", sorted(set(names)))
    assert sum(name.startswith("attention_decode") for name in names) == 5
    assert names.count("linear_attention[one token]") == 5 and names.count("gemm_silu_columns[skinny]") == 5
    assert names.count("add_parts_norm") == 1 + 9 + 1 - 1          # the scaled embedding, every later sublayer's read, the head
    engine.release(slot)
    close(last, want[299:], "bfloat16", record_property, "decoded", slack=2.0)
    engine32, _ = make(config, "float32", seed=3)
    slot = engine32.acquire()
    with ops.record_launches() as names:
        run(engine32, slot, tokens)
    assert "library_mm" not in names and "linear_attention[chunks]" not in names
    assert not any("tensor" in name or "tcgen05" in name or "skinny" in name or "mma" in name for name in names)


@pytest.mark.parametrize("softcap,sharp", [(None, 1.0), (50.0, 1.0), (8.0, 1.5), (1.5, 4.0)])
def test_every_form_of_the_bounded_sigmoid(softcap, sharp, record_property):
    """Scores as they are, and bounded scores that are small against the bound, of its size and far beyond it (the short
    polynomial, the long one and the exponential of the prompt kernel), at head widths 64 and 48, against the plain model;
    prompts and decoding give the same."""
    for dim in (64, 48):
        config = configs.single(configs.layer(configs.attention(4, 2, dim, dim, dim ** -0.5, chunk=170, softcap=softcap),
                                              configs.linear(1, 16, 16), left_scale=1.5, right_scale=0.2), width=64, groups=1)
        engine, tensors = make(config, "bfloat16", seed=3, sharp=sharp)
        tokens = prompt(config, 400, 5)
        want = plain(config, tensors, tokens)
        close(in_steps(engine, tokens, [400]), want, "bfloat16", record_property, f"whole {dim}")
        close(decoded(engine, tokens, 300), want, "bfloat16", record_property, f"decoded {dim}")


# ------------------------------------------------------------------ generation, the command line, the trace runner
def teacher_forced(config, tensors, request, tokens, bound):
    """(close calls, misses): tokens whose two best logits lie closer than the bound (either may be taken), and
    tokens that are not the plain model's choice although it was clear."""
    logits = plain(config, tensors, list(request) + list(tokens))[len(request) - 1:-1].numpy()
    close_calls = misses = 0
    for place, token in enumerate(tokens):
        row = logits[place]
        best, second = np.sort(row)[-1], np.sort(row)[-2]
        margin = bound * float(np.abs(row).max())
        if best - second >= margin:
            misses += token != int(np.argmax(row))
        else:
            close_calls += 1
            misses += row[token] < best - margin
    return close_calls, misses


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("use_graph", [True, False])
@pytest.mark.parametrize("name", sorted(configs.ALL))
def test_greedy_generation_through_the_engine(name, dtype, use_graph):
    """`Engine.generate`: batches of unequal prompts, decode steps replayed as a captured graph (with padding rows:
    three live sequences in four rows), slots reused by the next batch, prompts in portions."""
    config = configs.ALL[name]
    tensors = configs.tensors(config, 7)
    engine, _ = make(config, dtype, tensors=tensors, max_tokens=2048)
    requests = [prompt(config, n, 40 + n) for n in (5, 1, 70, 12, 33)]
    found = engine.generate(requests, max_new_tokens=12, ignore_eos=True, max_active=3, use_graph=use_graph)
    counts = [teacher_forced(config, tensors, r, t, GREEDY[dtype]) for r, t in zip(requests, found)]
    close_calls, misses = sum(c for c, _ in counts), sum(m for _, m in counts)
    # in bfloat16 a router's close call may fall the other way and cost that token
    assert all(len(tokens) == 12 for tokens in found) and close_calls <= 30 and misses <= (0 if dtype == "float32" else 2)
    again = engine.generate(requests[:2], max_new_tokens=12, ignore_eos=True, use_graph=use_graph)
    cut = engine.generate(requests, max_new_tokens=4, ignore_eos=True, use_graph=use_graph, prefill_chunk_size=16)
    if dtype == "float32":
        assert again == found[:2] and cut == [tokens[:4] for tokens in found]
    engine.cache.check()
    assert not engine.cache.slots.held
    engine.check_device_errors()


def write_folder(folder, config, tensors):
    from kidi_b200.weights.safetensors_io import write_safetensors
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(config))
    write_safetensors(str(folder / "model.safetensors"), tensors, metadata={"format": "pt"})


def test_the_command_line_generates(tmp_path, capsys):
    import kidi_b200
    config = configs.SMALL_A
    tensors = configs.tensors(config, 8)
    write_folder(tmp_path / "model", config, tensors)
    requests = [prompt(config, n, n) for n in (4, 19)]
    (tmp_path / "in.jsonl").write_text("".join(json.dumps({"token_ids": r, "id": str(i)}) + "\n"
                                              for i, r in enumerate(requests)))
    code = kidi_b200.main(["generate", "-m", str(tmp_path / "model"), "-i", str(tmp_path / "in.jsonl"), "-o",
                           str(tmp_path / "out.jsonl"), "--max-new-tokens", "6", "--ignore-eos", "--precision", "fp32"])
    assert code == 0, capsys.readouterr().err
    records = [json.loads(line) for line in (tmp_path / "out.jsonl").read_text().splitlines()]
    assert len(records) == 2
    for record in records:
        request = requests[int(record["id"])]
        assert teacher_forced(config, tensors, request, record["token_ids"], LARGEST["float32"]) == (0, 0)


def test_a_random_model_folder_runs(tmp_path):
    """`write_random_model` draws every tensor the design declares and the engine loads the folder it wrote."""
    import kidi_b200
    from safetensors import safe_open
    folder = kidi_b200.write_random_model(configs.SMALL_A, str(tmp_path / "model"), seed=3)
    engine = kidi_b200.Engine.load(folder, dtype="bfloat16", max_tokens=512)
    with safe_open(f"{folder}/model.safetensors", "pt") as handle:
        tensors = {name: handle.get_tensor(name) for name in handle.keys()}
    tokens = prompt(configs.SMALL_A, 80, 1)
    got, want = in_steps(engine, tokens, [80]), plain(configs.SMALL_A, tensors, tokens)
    assert float((got - want).abs().max()) < 0.1 * max(1.0, float(want.abs().max()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_trace_runner_replays_a_model_folder(tmp_path, dtype, record_property):
    """bin/trace_run on a Dibesun folder: three unequal requests start together (one of a single token), are decoded
    together until the shorter ones end, a step in which nothing is wanted, then a fourth request on what they gave
    back. `--max-tokens` is the tokens they hold, with no allowance for partly filled pages."""
    import os
    import subprocess
    import sys
    config = configs.SMALL_A
    tensors = configs.tensors(config, 9)
    write_folder(tmp_path / "model", config, tensors)
    a, b, c, d = (prompt(config, n, 60 + n) for n in (1, 75, 133, 90))
    want = {name: plain(config, tensors, tokens) for name, tokens in (("a", a), ("b", b), ("c", c), ("d", d))}
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a, "want": [0]}, {"id": "b", "tokens": b[:70], "want": [0, 69]},
                                     {"id": "c", "tokens": c[:129], "want": [5, 128]}], "end": ["a"]}]
    for index in range(5):
        entries = [{"id": "b", "tokens": [b[70 + index]], "want": [0] if index != 2 else []}]
        if index < 4:
            entries.append({"id": "c", "tokens": [c[129 + index]], "want": [0] if index != 2 else []})
        steps.append({"step": 1 + index, "entries": entries, "end": ["c"] if index == 3 else ["b"] if index == 4 else []})
    steps.append({"step": 6, "entries": [{"id": "d", "tokens": d, "want": [0, 45, 89]}], "end": ["d"]})
    out = tmp_path / "out"
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    result = subprocess.run(
        [sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path / "model"), "--dtype", dtype,
         "--out", str(out), "--max-tokens", str(1 + 75 + 133)],
        input="\n".join(json.dumps(step) for step in steps) + "\n", capture_output=True, text=True, timeout=900)
    assert result.returncode == 0, result.stderr
    assert result.stdout.split() == [word for step in steps for word in ("done", str(step["step"]))]
    read = lambda step: torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(-1, config["vocab"])).double()
    assert not (out / "3.f32").exists()                      # nothing was wanted in that step
    assert read(0).shape[0] == 5 and read(2).shape[0] == 2 and read(5).shape[0] == 1 and read(6).shape[0] == 3
    close(torch.cat([read(0), read(2), read(5), read(6)]),
          torch.cat([torch.stack([want["a"][0], want["b"][0], want["b"][69], want["c"][5], want["c"][128]]),
                     torch.stack([want["b"][71], want["c"][130]]), want["b"][74:75], want["d"][[0, 45, 89]]]),
          dtype, record_property, "prompts together, decoded together, the last one alone, on reused pages", slack=2.0)


# ------------------------------------------------------------------ routed experts on prompts
@pytest.mark.parametrize("gated", [True, False])
@pytest.mark.parametrize("rows,experts,top,hidden,inter", [(200, 6, 2, 64, 24), (700, 16, 3, 136, 72), (300, 5, 5, 256, 200),
                                                           (129, 40, 1, 48, 136)])
def test_products_over_groups_of_experts(rows, experts, top, hidden, inter, gated, monkeypatch):
    """Slots grouped on the device (an expert that nobody chooses, one that most choose), the product over groups with and
    without the gate, and the routed feed-forward as a whole against its form with the slots sorted on the host."""
    from kidi_b200.kernels import ops, routed, tcgen05
    generator = torch.Generator().manual_seed(rows)
    bias = torch.randn(experts, generator=generator)
    bias[experts // 2] += 6.0
    bias[0] -= 60.0 if top < experts else 0.0
    chosen = torch.topk(torch.randn(rows, experts, generator=generator) + bias, top).indices.int()
    source, place, tiles = (t.cpu() for t in routed.group_slots(chosen.cuda(), experts))
    flat = chosen.reshape(-1)
    assert torch.equal(source[place.long()], torch.arange(rows * top, dtype=torch.int32))      # every slot has its row
    assert int((source >= 0).sum()) == rows * top and source.numel() % 128 == 0
    assert torch.equal(tiles[place.long() // 128], flat)                                      # in a tile of its expert
    used = (torch.bincount(flat, minlength=experts) + 127) // 128
    assert torch.equal(torch.bincount(tiles[tiles >= 0], minlength=experts), used) and int((tiles < 0).sum()) == tiles.numel() - int(used.sum())
    x = torch.randn(source.numel(), hidden, generator=generator).bfloat16()
    weight = (torch.randn(experts, (2 if gated else 1) * inter, hidden, generator=generator) / hidden ** 0.5).bfloat16()
    got = tcgen05.gemm_grouped(x.cuda(), weight.cuda(), tiles.cuda(), gated).double().cpu()
    for tile, expert in enumerate(tiles.tolist()):
        if expert < 0:
            continue
        y = x[128 * tile:128 * tile + 128].double() @ weight[expert].double().t()
        want = plain_dibesun.silu(y[:, :inter]) * y[:, inter:] if gated else y
        assert torch.allclose(got[128 * tile:128 * tile + 128], want, atol=2e-2, rtol=2e-2)


def test_routed_prompts_grouped_on_the_device_and_sorted_on_the_host(monkeypatch, record_property):
    """The same prompt through both forms of the routed feed-forward: each names its kernels, the logits agree within
    bfloat16 rounding, and a request in a batch is what it is alone."""
    from kidi_b200 import StepBatch
    from kidi_b200.kernels import ops
    from kidi_b200.parts import routed as part
    config = configs.single(configs.layer(configs.attention(2, 1, 16, 16, 0.3, softcap=20.0), configs.linear(4, 16, 16),
                                          configs.routed(6, 2, 40, shared=24)), width=64, groups=2)
    engine, tensors = make(config, "bfloat16", seed=3)
    a, b = prompt(config, 300, 1), prompt(config, 120, 2)
    found = {}
    for grouped in (True, False):
        monkeypatch.setattr(part, "GROUPED", grouped)
        with ops.record_launches() as names:
            found[grouped] = in_steps(engine, a, [300])
        assert ("group_slots" in names and "gemm_silu_gate[tcgen05, groups]" in names) == grouped
        assert ("library_bmm" in names) == (not grouped)
        close(found[grouped], follow(engine, 0, "bfloat16", config, tensors, a, None), "bfloat16", record_property, str(grouped))
    monkeypatch.setattr(part, "GROUPED", True)
    slots = [engine.acquire(), engine.acquire()]
    both = engine.step(StepBatch(slots, [b, a], [[], list(range(300))])).double().cpu()
    assert float((both - found[True]).abs().max()) < 0.05 * float(both.abs().max())
    engine.check_device_errors()
