"""Bimolix on the GPU against the plain implementation (tests/plain_bimolix.py, float64, whole sequences): each mechanism
alone (retention by the scan, in chunks and token by token with its rotation and its finish, attention whose values are its
keys with a number per distance, a one in the denominator and a gate per element in every kernel that has it, the norms and
the cache write before it, the router with its correction, groups and the shared expert's gate, bounded gates, one layer
against plain models with one constant or one rule changed), whole prompts, prompts then token-by-token decoding across page
and chunk borders, portions down to two tokens, batches of unequal requests against each alone, slots and pages that are used
again, keys that stand out just inside and just outside a chunk (in prompts and decoded), the first tokens of a sequence,
layers that run with another layer's tensors, long decoding, and greedy generation through `Engine.generate`, the command
line and the trace runner. Weights and configurations are the tests' own (tests/bimolix_configs.py)."""
import copy
import json
import types

import numpy as np
import pytest
import torch

import bimolix_configs as configs
import plain_bimolix

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
    return plain_bimolix.forward(config, tensors, tokens, dtype=torch.float64, choices=choices, margin=CLOSE_CALL)


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
def paged(generator, slots, pages_per, kv_heads, dim, dtype, ring=0):
    """An empty cache of keys alone with scrambled pages."""
    keys = torch.zeros(slots * pages_per, kv_heads, 64, dim, dtype=dtype).cuda()
    table = torch.randperm(slots * pages_per, generator=generator).reshape(slots, pages_per).int()
    return types.SimpleNamespace(keys=keys, values=keys[..., :0], table=table.cuda(), page_size=64, ring_pages=ring)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,dim,ring", [(4, 2, 16, 0), (3, 1, 10, 0), (32, 8, 128, 0), (6, 3, 24, 2), (8, 2, 64, 1)])
def test_keys_before_their_norm_go_to_the_cache(dtype, heads, kv_heads, dim, ring):
    """Queries normed with the product of both weights; keys left as they are, in the cache's pages (or not, beyond a ring's
    reach), and with their norm but without a weight in a matrix of their own; a padding row and the columns behind the keys
    left alone; a copy alone."""
    from kidi_b200.kernels import ops
    generator = torch.Generator().manual_seed(heads)
    lengths, starts, slots = (70, 3), (60, 0), (2, 0)
    rows, width, pages_per = sum(lengths), (heads + kv_heads) * dim, ring or 3
    qkv = torch.randn(rows, width + 8 + (-width % 8), generator=generator).to(dtype)
    weight = torch.randn(dim, generator=generator) * 0.3 + 1
    tables = step_tables(lengths, starts, slots)
    tables.row_seq[72] = -1
    view = paged(generator, 3, pages_per, kv_heads, dim, dtype, ring)
    held, normed = qkv.cuda(), torch.zeros(rows, kv_heads * dim, dtype=dtype).cuda()
    common = dict(heads=heads, kv_heads=kv_heads, head_dim=dim, k_norm=None, eps=1e-5, cos=None, sin=None, rotary_dim=0,
                  tables=tables, kv_view=view, tied=True)
    ops.rope_store(held, q_norm=weight.cuda(), store=False, k_normed=normed, **common)
    assert not view.keys.any()
    ops.rope_store(held, q_norm=None, store=True, transform=False, **common)
    split = heads * dim
    want = plain_bimolix.by_rms(qkv[:, :split].double().reshape(rows, heads, dim), 1e-5) * weight.double()
    keys = plain_bimolix.by_rms(qkv[:, split:width].double().reshape(rows, kv_heads, dim), 1e-5)
    live = [row for row in range(rows) if row != 72]
    loose = 1e-5 if dtype == torch.float32 else 3e-2
    assert torch.allclose(held[live, :split].double().cpu(), want.reshape(rows, -1)[live], atol=loose)
    assert torch.allclose(normed[live].double().cpu(), keys.reshape(rows, -1)[live], atol=loose) and not normed[72].any()
    assert torch.equal(held[:, split:].cpu(), qkv[:, split:]) and torch.equal(held[72].cpu(), qkv[72])
    at = 0
    for b, (count, start) in enumerate(zip(lengths, starts)):
        for t in range(count):
            row, position = at + t, start + t
            if ring and position < start + count - 64 * ring:
                continue                                        # a later token of the step took its place
            stored = view.keys[view.table[slots[b], (position // 64) % pages_per].long(), :, position % 64].cpu().reshape(-1)
            assert torch.equal(stored, torch.zeros_like(stored) if row == 72 else qkv[row, split:width])
        at += count


def test_the_distance_bias_lies_where_the_kernels_look():
    from kidi_b200.kernels import ops
    by_distance = torch.randn(37, 3, generator=torch.Generator().manual_seed(1))
    bias = ops.DistanceBias(by_distance.cuda())
    address, stride, last = bias.fields(3)
    assert address == bias.table.data_ptr() + 4 * bias.BEFORE and last == 36 and stride == bias.table.shape[1]
    address, copy_, origin, last = bias.descending(3)
    assert address % 16 == 0 and copy_ % 4 == 0 and last == 36
    copies = bias.copies.cpu()
    for distance in (-bias.BEFORE, -5, 0, 1, 17, 36, 37, 200, 36 + bias.BEHIND):
        want = by_distance[min(distance, 36)] * 1.4426950408889634 if distance >= 0 else torch.zeros(3)
        assert torch.allclose(bias.table_log2[:, bias.BEFORE + distance].cpu(), want)
        for shift in range(4):
            assert torch.allclose(copies[:, shift, origin - distance + shift], want)


def tied_attention(q, keys, scale, eps, bias, chunk, positions, gate):
    """Row r (at `positions[r]`) of one sequence: q [rows, H, d] with both norm weights in it, keys [T, G, d] before their
    norm, bias [n, H] by distance; sums over the keys of its chunk up to itself, times sigmoid(gate)."""
    H, G = q.shape[1], keys.shape[1]
    normed = plain_bimolix.by_rms(keys, eps)
    out = torch.zeros_like(q)
    for r, p in enumerate(positions):
        first = p - p % chunk if chunk else 0
        back = (p - torch.arange(first, p + 1)).clamp(max=bias.shape[0] - 1)
        for h in range(H):
            g = h // (H // G)
            s = normed[first:p + 1, g] @ q[r, h] * scale + bias[back, h]
            weights = plain_bimolix.softmax_with_one(s[None], torch.ones(1, len(s), dtype=torch.bool))[0]
            out[r, h] = weights @ keys[first:p + 1, g]
    return out.reshape(len(positions), -1) * torch.sigmoid(gate)


def attention_step(lengths, starts):
    as_np = lambda values: np.asarray(values, dtype=np.int32)
    spaces = {}

    def workspace(name, count, zero=False):
        if name not in spaces or spaces[name].numel() < count:
            spaces[name] = torch.zeros(count, dtype=torch.float32).cuda()
        return spaces[name]

    plan = types.SimpleNamespace(is_decode=all(n == 1 for n in lengths), n_seqs=len(lengths), max_new=max(lengths),
                                 max_total=max(n + s for n, s in zip(lengths, starts)), seq_start=as_np(starts))
    return types.SimpleNamespace(plan=plan, tables=step_tables(lengths, starts, list(range(len(lengths)))), workspace=workspace)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,dim,chunk,entries", [
    (8, 2, 128, None, 300), (4, 2, 64, 150, 40), (2, 2, 64, 64, 3), (3, 1, 48, 100, 90), (12, 1, 32, 130, 600), (5, 1, 16, 1, 1),
    (40, 2, 32, 90, 20), (3, 3, 20, 77, 50)])
def test_attention_whose_values_are_its_keys(heads, kv_heads, dim, chunk, entries, dtype, record_property):
    """Prompts (every key in the step; continued from pages; continued from a ring, where there are chunks) and single tokens
    through every form of the decode kernel, with a number per distance, a one in the denominator and a gate per element. A
    few keys are made long (their norm takes that back, their value does not)."""
    from kidi_b200.kernels import attention, ops
    generator = torch.Generator().manual_seed(dim + heads)
    draw = lambda *shape: torch.randn(*shape, generator=generator)
    lengths, eps, scale = (333, 70, 1), 1e-4, 0.8 * dim ** -0.5
    bias = draw(entries, heads) * 1.5
    table = ops.DistanceBias(bias.cuda())
    sinks = torch.zeros(heads).cuda()
    q, keys, gates = [], [], []
    for n in lengths:
        keys.append((draw(n, kv_heads, dim) * torch.exp(draw(n, kv_heads, 1))).to(dtype))
        q.append((draw(n, heads, dim) * 2).to(dtype))
        gates.append(draw(n, heads * dim).to(dtype))
    want = [tied_attention(a.double(), k.double(), scale, eps, bias.double(), chunk, range(len(a)), g.double())
            for a, k, g in zip(q, keys, gates)]
    loose = 2e-5 if dtype == torch.float32 else 2e-2
    launcher = attention.AttentionLauncher(heads=heads, kv_heads=kv_heads, head_dim=dim, scale=scale, chunk=chunk, tied=True,
                                           biased=True, key_eps=eps)
    extras = dict(sinks=sinks, distance_bias=table)

    def rows_of(spans):
        """Packed rows [q | k | gate] of tokens spans[b] of each sequence."""
        pieces = [torch.cat([q[b][s].reshape(-1, heads * dim), keys[b][s].reshape(-1, kv_heads * dim), gates[b][s]], 1)
                  for b, s in enumerate(spans)]
        packed = torch.cat(pieces).cuda()
        pad = -packed.shape[1] % 8
        return torch.cat([packed, packed.new_zeros(packed.shape[0], pad)], 1) if pad else packed

    def compare(out, spans, what):
        expected = torch.cat([w[s] for w, s in zip(want, spans)])
        error = float((out.double().cpu() - expected).norm() / expected.norm())
        worst = float((out.double().cpu() - expected).abs().max() / expected.abs().max())
        record_property(what, (error, worst))
        assert error < loose and worst < 2 * loose, (what, error, worst)

    def gate_of(qkv):
        at = (heads + kv_heads) * dim
        return qkv[:, at:at + heads * dim]

    def view_for(held, ring):
        """A cache that holds the first held[b] tokens of each sequence."""
        view = paged(generator, len(lengths), ring or 6, kv_heads, dim, dtype, ring)
        for b, count in enumerate(held):
            for u in range(max(0, count - 64 * ring) if ring else 0, count):
                view.keys[view.table[b, (u // 64) % (ring or 6)].long(), :, u % 64] = keys[b][u].cuda()
        return view

    ring = -(-chunk // 64) if chunk else 0
    whole = [slice(0, n) for n in lengths]
    # (1) whole prompts: every key is a row of the step
    step = attention_step(lengths, (0, 0, 0))
    qkv = rows_of(whole)
    out = torch.empty(qkv.shape[0], heads * dim, dtype=dtype).cuda()
    normed = None
    if launcher.wants_normed_keys(step.plan, qkv):
        normed = plain_bimolix.by_rms(torch.cat(keys).double(), eps).to(dtype).reshape(qkv.shape[0], -1).cuda()
    with ops.record_launches() as names:
        launcher.run(step, qkv, out, kv_view=None, keys_in_step=True, element_gate=gate_of(qkv), k_normed=normed, **extras)
    tensor_core = dtype == torch.bfloat16 and dim % 16 == 0
    assert names == (["attention"] if not tensor_core else ["attention_prefill_tcgen05"] if dim in (64, 128)
                     else ["attention_prefill[mma.sync]"])
    compare(out, whole, "whole")
    # (2) the last tokens as a portion that continues what the cache holds (its own rows read from the step)
    for cut, rings in (((200, 5, 0), (0, ring)), ((331, 68, 0), (ring,))):
        for pages in dict.fromkeys(rings):
            spans = [slice(c, n) for c, n in zip(cut, lengths)]
            step = attention_step([n - c for c, n in zip(cut, lengths)], cut)
            qkv = rows_of(spans)
            out = torch.empty(qkv.shape[0], heads * dim, dtype=dtype).cuda()
            launcher.run(step, qkv, out, kv_view=view_for(cut, pages), keys_in_step=True, element_gate=gate_of(qkv), **extras)
            compare(out, spans, f"portion from {cut[0]}, ring of {pages}")
    # (3) the last token alone, its key in the cache already, in every form of the decode kernel
    spans = [slice(n - 1, n) for n in lengths]
    step = attention_step((1, 1, 1), [n - 1 for n in lengths])
    qkv = rows_of(spans)
    for pages in dict.fromkeys((0, ring)):
        view = view_for(lengths, pages)
        for splits in (None, 1, 2, 3, 5):
            out = torch.empty(3, heads * dim, dtype=dtype).cuda()
            launcher.run(step, qkv, out, kv_view=view, keys_in_step=False, element_gate=gate_of(qkv), splits=splits, **extras)
            compare(out, spans, f"decoded, {splits} splits, ring of {pages}")
    # (4) the same where the kernel norms the query and stores the key itself
    rotation = dict(q_norm=torch.full((dim,), 1.25).cuda(), k_norm=None, cos=None, sin=None, rotary_dim=0)
    probe = view_for([n - 1 for n in lengths], ring)
    if launcher.fuses_rotation(step.plan, qkv, kv_view=probe, **rotation):
        for b in range(3):
            a = plain_bimolix.by_rms(q[b][-1:].double(), eps) * 1.25
            want[b][-1:] = tied_attention(a, keys[b].double(), scale, eps, bias.double(), chunk, [lengths[b] - 1], gates[b][-1:].double())
        for splits in (None, 1, 2, 5):
            view = view_for([n - 1 for n in lengths], ring)
            out = torch.empty(3, heads * dim, dtype=dtype).cuda()
            launcher.run(step, qkv, out, kv_view=view, keys_in_step=False, element_gate=gate_of(qkv), splits=splits,
                         rotation=dict(rotation, eps=eps, store=True), **extras)
            compare(out, spans, f"decoded with its norm, {splits} splits")
            for b, n in enumerate(lengths):
                stored = view.keys[view.table[b, ((n - 1) // 64) % (ring or 6)].long(), :, (n - 1) % 64].cpu()
                assert torch.equal(stored, keys[b][-1])
    else:
        assert not tensor_core or heads // kv_heads > 8
    assert attention.timeout_flags() == 0


@pytest.mark.parametrize("form", ["scan", "chunks", "bits"])
@pytest.mark.parametrize("heads,dim,vdim,rot", [(3, 16, 48, 16), (2, 32, 64, 32), (5, 48, 16, 20), (2, 128, 128, 128), (3, 80, 32, 6),
                                                (2, 64, 64, 0), (2, 16, 16, 14)])
def test_retention_in_portions(heads, dim, vdim, rot, form, monkeypatch):
    """The scan, the chunked tensor-core form and the one-token kernel against the loop over each sequence (decays of 0
    and 1 among them), whole and partly rotated heads at late positions, with states that are carried in and slots in any
    order: portions that are whole chunks, a token more and less than one, single tokens; the finish head by head; the scan's
    results do not depend on the cut."""
    from kidi_b200.kernels import linear_attention as kernels
    from kidi_b200.kernels import ops
    dtype = torch.float32 if form == "bits" else torch.bfloat16
    monkeypatch.setattr(kernels, "MIN_CHUNKED_TOKENS", 2 if form == "chunks" else 0)
    generator = torch.Generator().manual_seed(dim + rot)
    lengths, slots, late, eps, scale = (200, 1, 131), (2, 0, 4), 400, 1e-3, dim ** -0.5
    total, width = sum(lengths), heads * (2 * dim + 2 * vdim)
    packed = torch.randn(total, width + 8, generator=generator).to(dtype)
    decay = torch.tensor(([0.0, 1.0] + [0.9 + 0.02 * h for h in range(heads)])[:heads])
    start = torch.randn(6, heads, dim, vdim, generator=generator)
    angle = torch.arange(late + 200, dtype=torch.float64)[:, None] * (50.0 ** (-2.0 * torch.arange(rot // 2, dtype=torch.float64) / max(rot, 1)))
    cos, sin = (torch.cos(angle).float().contiguous().cuda(), torch.sin(angle).float().contiguous().cuda()) if rot else (None, None)
    qk, values = heads * dim, heads * vdim
    parts = lambda x: (x[:, :qk], x[:, qk:2 * qk], x[:, 2 * qk:2 * qk + values], x[:, 2 * qk + values:width])
    want, states, at = [], [], 0
    for b, count in enumerate(lengths):
        q, k, v, g = (x[at:at + count].double().reshape(count, heads, -1) for x in parts(packed))
        S = start[slots[b]].double().clone()
        read = plain_bimolix.fixed_decay_recurrence(plain_bimolix.rotate(q, rot, 50.0, late) if rot else q,
                                                    (plain_bimolix.rotate(k, rot, 50.0, late) if rot else k) * scale, v, decay.tolist(), S)
        want.append((plain_bimolix.by_rms(read, eps) * plain_bimolix.silu(g)).reshape(count, -1))
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
                q, k, v, g = parts(packed[rows].cuda())
                out = torch.empty(len(rows), values, dtype=dtype).cuda()
                kernels.retention(q, k, v, g, decay.cuda(), state, out, heads=heads, dim=dim, vdim=vdim,
                                  tables=step_tables(sizes, [late + done[b] for b in live], [slots[b] for b in live]),
                                  seqs=len(live), one_token=max(sizes) == 1, longest=max(sizes), cos=cos, sin=sin, rotary_dim=rot,
                                  key_scale=scale, eps=eps, silu=True)
                out, at = out.cpu(), 0
                for b, n in zip(live, sizes):
                    pieces[b].append(out[at:at + n])
                    at += n
                    done[b] += n
        assert ("retention[chunks]" if form == "chunks" else "scalar_recurrence") in names
        if cuts[0] == 199:
            assert "retention[one token]" in names
        found.append([torch.cat(p) for p in pieces])
        for b in range(len(lengths)):
            error = float((found[-1][b].double() - want[b]).abs().max() / want[b].abs().max())
            assert error < (2e-5 if dtype == torch.float32 else 6e-3), (cuts, b, error)
            scale_of = float(states[b].abs().max())
            assert float((state[slots[b]].double().cpu() - states[b]).abs().max()) < 4e-6 * scale_of, (cuts, b)
        untouched = [slot for slot in range(6) if slot not in slots]
        assert torch.equal(state[untouched].cpu(), start[untouched])
    if form == "bits":
        assert all(torch.equal(a, b) for cut in found[1:4] for a, b in zip(cut, found[0]))


def test_wide_heads_of_retention_take_what_fits(monkeypatch):
    """Heads of 256 x 256 (the chunked form at the edge of shared memory), values too wide for one cluster, heads of a step in
    groups."""
    from kidi_b200.kernels import linear_attention as kernels
    from kidi_b200.kernels import ops
    generator = torch.Generator().manual_seed(8)
    for heads, dim, vdim, floats, length in ((1, 256, 256, 1 << 30, 150), (3, 64, 320, 1 << 30, 40), (5, 32, 64, 1, 150)):
        monkeypatch.setattr(kernels, "SCRATCH_FLOATS", floats)
        q, k, v, g = (torch.randn(length, heads * n, generator=generator).bfloat16() for n in (dim, dim, vdim, vdim))
        decay = torch.rand(heads, generator=generator) * 0.2 + 0.8
        S = torch.zeros(heads, dim, vdim, dtype=torch.float64)
        shaped = [x.double().reshape(length, heads, -1) for x in (q, k, v)]
        want = plain_bimolix.by_rms(plain_bimolix.fixed_decay_recurrence(shaped[0], shaped[1] * 0.3, shaped[2], decay.tolist(), S), 1e-4)
        want = want.reshape(length, -1) * torch.sigmoid(g.double())
        state = torch.zeros(2, heads, dim, vdim).cuda()
        rows = []
        with ops.record_launches() as names:
            for begin, end in ((0, length - 1), (length - 1, length)):
                out = torch.empty(end - begin, heads * vdim, dtype=torch.bfloat16).cuda()
                kernels.retention(*(x[begin:end].cuda() for x in (q, k, v, g)), decay.cuda(), state, out, heads=heads, dim=dim,
                                  vdim=vdim, tables=step_tables([end - begin], [begin], [1]), seqs=1, one_token=end - begin == 1,
                                  longest=end - begin, cos=None, sin=None, rotary_dim=0, key_scale=0.3, eps=1e-4, silu=False)
                rows.append(out.cpu())
        assert names.count("retention[chunks]") == (0 if vdim > 256 else heads if floats == 1 else 1)
        assert ("retention[one token]" in names) == (vdim <= 256)
        assert float((torch.cat(rows).double() - want).abs().max() / want.abs().max()) < 6e-3
        assert float((state[1].double().cpu() - S).abs().max() / S.abs().max()) < 4e-6


def test_a_padding_sequence_leaves_the_state_alone():
    """One-token steps: a padding sequence in front of live ones, widths with and without 16-byte pieces."""
    from kidi_b200.kernels import linear_attention as kernels
    for dtype in (torch.float32, torch.bfloat16):
        for heads, dim, vdim, rot in ((2, 7, 5, 6), (3, 256, 36, 64), (1, 130, 33, 0), (4, 16, 256, 16)):
            generator = torch.Generator().manual_seed(dim)
            q, k, v, g = (torch.randn(3, heads * n, generator=generator).to(dtype) for n in (dim, dim, vdim, vdim))
            decay = torch.rand(heads, generator=generator)
            start = torch.randn(4, heads, dim, vdim, generator=generator)
            state, tables = start.clone().cuda(), step_tables([1, 1, 1], [9, 0, 3], [2, 3, 0])
            tables.row_seq[1] = -1
            angle = torch.rand(20, max(rot // 2, 1), generator=generator) * 6
            cos, sin = (torch.cos(angle).cuda(), torch.sin(angle).cuda()) if rot else (None, None)
            out = torch.zeros(3, heads * vdim, dtype=dtype).cuda()
            kernels.retention(q.cuda(), k.cuda(), v.cuda(), g.cuda(), decay.cuda(), state, out, heads=heads, dim=dim, vdim=vdim,
                              tables=tables, seqs=3, one_token=True, longest=1, cos=cos, sin=sin, rotary_dim=rot, key_scale=0.5,
                              eps=1e-4, silu=True)
            for b, slot, position in ((0, 2, 9), (2, 0, 3)):
                def turned(x):
                    x = x[b].double().reshape(1, heads, dim)
                    if not rot:
                        return x
                    c, s = torch.cos(angle.double())[position], torch.sin(angle.double())[position]
                    u, w = x[..., :rot // 2], x[..., rot // 2:rot]
                    return torch.cat([u * c - w * s, w * c + u * s, x[..., rot:]], -1)
                S = start[slot].double()
                read = plain_bimolix.fixed_decay_recurrence(turned(q), turned(k) * 0.5, v[b:b + 1].double().reshape(1, heads, vdim),
                                                            decay.tolist(), S)
                want = (plain_bimolix.by_rms(read, 1e-4).reshape(-1) * plain_bimolix.silu(g[b].double()))
                assert torch.allclose(out[b].double().cpu(), want, atol=1e-4 if dtype == torch.float32 else 3e-2, rtol=1e-2)
                assert torch.allclose(state[slot].double().cpu(), S, atol=1e-5)
            assert torch.equal(state[[1, 3]].cpu(), start[[1, 3]]) and not out[1].any()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_a_norm_and_a_gate_head_by_head(dtype):
    from kidi_b200.kernels import linear_attention as kernels
    generator = torch.Generator().manual_seed(3)
    for rows, heads, width, silu, weighted in ((3, 5, 9, True, False), (2, 1, 64, False, True), (4, 16, 128, True, True)):
        read = torch.randn(rows, heads * width, generator=generator) * 5
        weight = torch.randn(heads * width, generator=generator) * 0.3 + 1 if weighted else None
        gate = (torch.randn(rows, heads * width + 8, generator=generator) * 2).to(dtype)
        out = torch.zeros(rows, heads * width + 16, dtype=dtype).cuda()
        kernels.head_norm_gate(read.cuda(), weight.cuda() if weighted else None, gate.cuda()[:, 8:], heads, 1e-5, -0.6, silu,
                               out[:, 8:8 + heads * width])
        z = gate[:, 8:].double()
        want = -0.6 * plain_bimolix.by_rms(read.double().reshape(rows, heads, width), 1e-5).reshape(rows, -1) \
            * (plain_bimolix.silu(z) if silu else torch.sigmoid(z)) * (weight.double() if weighted else 1.0)
        loose = dict(atol=2e-5, rtol=1e-5) if dtype == torch.float32 else dict(atol=2e-2, rtol=1e-2)
        assert torch.allclose(out[:, 8:8 + heads * width].double().cpu(), want, **loose)
        assert not out[:, :8].any() and not out[:, 8 + heads * width:].any()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_router_with_a_correction_and_ranked_groups(dtype):
    """The correction counts in the choice of experts and groups and not in the weights; groups by their two best (also groups
    of one); all scores negative; weights over their sum, times a number; the shared expert's gate beside them."""
    from kidi_b200.kernels import routed
    generator = torch.Generator().manual_seed(5)
    for experts, top, groups, keep, shift in ((6, 2, 3, 2, 0.0), (16, 4, 4, 2, 0.0), (40, 7, 8, 3, -5.0), (8, 3, 8, 5, -2.0), (12, 12, 1, 1, 0.0),
                                              (33, 5, 3, 1, 0.0), (17, 4, 1, 1, -3.0)):
        x = torch.randn(9, 72, generator=generator).to(dtype)
        router = (torch.randn(experts, 72, generator=generator) * 0.3).to(dtype)
        row = (torch.randn(1, 72, generator=generator) * 0.3).to(dtype)
        correction = torch.randn(experts, generator=generator) * 0.4 + shift
        share = torch.empty(9).cuda()
        chosen, weight = routed.route(x.cuda(), router.cuda(), top, True, "sigmoid", groups, keep, 1e-20,
                                      correction=correction.cuda(), two_largest=True, weight_scale=1.7, share_row=row.cuda(), share=share)
        s = torch.sigmoid(x.double() @ router.double().t())
        for r in range(9):
            want = plain_bimolix.router_choice(s[r] + correction.double(), top, groups, keep)
            assert torch.equal(chosen[r].cpu().long(), want)
            assert torch.allclose(weight[r].double().cpu(), s[r, want] / s[r, want].sum() * 1.7, atol=1e-5)
        assert torch.allclose(share.double().cpu(), torch.sigmoid(x.double() @ row[0].double()), atol=1e-5)
    # many rows (four a block, the last block short of one): what a few rows give, bit for bit
    x, router = torch.randn(1027, 72, generator=generator).to(dtype).cuda(), (torch.randn(12, 72, generator=generator) * 0.3).to(dtype).cuda()
    correction, row = (torch.randn(12, generator=generator) * 0.4).cuda(), (torch.randn(1, 72, generator=generator) * 0.3).to(dtype).cuda()

    def route(some):
        share = torch.empty(some.shape[0]).cuda()
        chosen, weight = routed.route(some.contiguous(), router, 3, True, "sigmoid", 4, 2, 1e-20, correction=correction,
                                      two_largest=True, weight_scale=0.7, share_row=row, share=share)
        return chosen.float(), weight, share

    whole, pieces = route(x), [route(piece) for piece in x.split(100)]
    for index in range(3):
        assert torch.equal(whole[index], torch.cat([piece[index] for piece in pieces]))


@pytest.mark.parametrize("rows,experts,top,hidden,inter", [(3, 5, 2, 64, 24), (200, 6, 2, 64, 24), (300, 5, 5, 136, 72), (40, 4, 3, 50, 22)])
def test_bounded_gates_in_every_form(rows, experts, top, hidden, inter, monkeypatch, record_property):
    """Routed experts with bounded gates through the choice, grouped on the device and sorted on the host, in both precisions,
    with a shared expert of other limits under a gate of one number a token: against the plain sum. Limits that bind."""
    from kidi_b200.kernels import ops
    from kidi_b200.parts import routed as part
    from kidi_b200.parts.base import BuildEnv
    from kidi_b200.parts.spec import PartSpec
    generator = torch.Generator().manual_seed(rows)
    mlp = configs.routed(experts, top, inter, limit=0.8, scale=1.3, shared=inter + 8, shared_limit=1.4)
    config = configs.single(configs.layer(configs.retention(1, 8, 8), mlp), width=hidden)
    w = configs.tensors(config, 3)
    h = torch.randn(rows, hidden, generator=generator)
    for dtype in (torch.float32, torch.bfloat16):
        cast = {name[len("l0.mlp."):]: t.to(dtype).cuda() for name, t in w.items() if name.startswith("l0.mlp.")}
        built = part.RoutedExperts(PartSpec("routed_experts", {
            "hidden_size": hidden, "expert_size": inter, "experts": experts, "top": top, "score": "sigmoid", "renormalise": True,
            "renormalise_eps": 1e-20, "weight_on": "output", "correction_name": "correction", "weight_scale": 1.3,
            "group_score": "two_largest", "activation": "bounded_swish", "limit": 0.8, "shared_size": inter + 8, "shared_limit": 1.4,
            "shared_gate_name": "sg"}), BuildEnv(dtype=dtype, device=torch.device("cuda:0"), max_positions=8))
        for name, each in (("experts.gate_up", ("gate", "up")), ("experts.down", ("down",))):
            cast[name] = torch.cat([cast[f"e{e}.{piece}"] for e in range(experts) for piece in each])
        cast["shared.gate_up"] = torch.cat([cast["shared.gate"], cast["shared.up"]])
        built.bind(cast)
        x = h.to(dtype).cuda()
        ctx = types.SimpleNamespace(plan=types.SimpleNamespace(is_decode=False))
        forms = [True, False] if dtype == torch.bfloat16 else [True]
        for grouped in forms:
            monkeypatch.setattr(part, "GROUPED", grouped)
            with ops.record_launches() as names:
                got = built.forward(x, ctx)
            chosen = plain_choice(x, w, mlp, experts)
            want = plain_bimolix.routed(x.double().cpu(), {n: t.double() for n, t in w.items()}, "l0.mlp.", mlp, chosen, 0.02)
            error = float((got.double().cpu() - want).norm() / want.norm())
            record_property(f"{dtype}, grouped {grouped}", (error, sorted(set(names))))
            assert error < (1e-5 if dtype == torch.float32 else 1.5e-2), (dtype, grouped, error)
            if dtype == torch.bfloat16 and rows * top > part.SLOT_PATH_MAX and hidden % 8 == 0:
                assert ("gemm_bounded_gate[tcgen05, groups]" in names) == grouped and ("library_bmm" in names) == (not grouped)
            elif rows <= 8 and dtype == torch.bfloat16:
                assert "gemm_bounded_gate[skinny]" in names and "expert_slots" in names


def plain_choice(x, w, mlp, experts):
    from kidi_b200.kernels import routed
    groups = mlp["router"].get("groups") or {"count": 1, "keep": 1}
    return routed.route(x, w["l0.mlp.router"].to(x.dtype).cuda(), mlp["router"]["top"], True, "sigmoid", groups["count"], groups["keep"],
                        1e-20, correction=w["l0.mlp.correction"].float().cuda(), two_largest=True)[0].cpu()


# ------------------------------------------------------------------ one layer
MIX = ("layers", 0, "mixer")
MLP = ("layers", 0, "mlp")
ONE_ATTENTION = configs.layer(configs.attention(4, 2, 16, 0.4, 50, chunk=70),
                              configs.routed(8, 3, 24, limit=0.9, scale=1.6, groups=(4, 2), shared=16, shared_limit=0.7))
ONE_RETENTION = configs.layer(configs.retention(3, 16, 20, (0.6, 0.95, 0.999), rot=12, base=500.0), configs.dense(40))
# what must not be confused with what: (path into the configuration, other value); None removes the key; a pair of values:
# the finer one for 32-bit, the coarser one where bfloat16 rounding would drown the finer
OTHERS = {
    "attention": [(MIX + ("mask", "size"), 69), (MIX + ("mask", "size"), 71), (MIX + ("mask",), None), (MIX + ("scale",), (0.38, 0.2)),
                  (MIX + ("bias_max",), (51, 90)), (("norm", "eps"), (1e-4, 0.3)), (MLP + ("router", "top"), 2),
                  (MLP + ("router", "scale"), (1.5, 0.8)), (MLP + ("router", "groups"), None), (MLP + ("router", "groups", "keep"), 3),
                  (MLP + ("expert", "limit"), (0.85, 0.4)), (MLP + ("shared", "limit"), (0.75, 2.0)), (MLP + ("shared",), None)],
    "retention": [(MIX + ("decay",), [0.95, 0.6, 0.999]), (MIX + ("decay",), [0.6, 0.95, 0.98]), (MIX + ("rot", "dims"), 16),
                  (MIX + ("rot", "dims"), 10), (MIX + ("rot", "base"), (480.0, 100.0)), (("norm", "eps"), (1e-4, 0.3)),
                  (MLP, None)]}


def other_rules(monkeypatch, config, tensors, tokens, kind):
    """Plain models with one rule changed."""
    found = []

    def with_patch(name, replacement):
        with monkeypatch.context() as patch:
            patch.setattr(plain_bimolix, name, replacement)
            found.append(plain(config, tensors, tokens))

    def without(*names, value=0.0):
        found.append(plain(config, {name: torch.full_like(t, value) if name.endswith(names) else t for name, t in tensors.items()}, tokens))

    T = len(tokens)
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    with_patch("stream_norm", lambda x, weight, eps: plain_bimolix.by_rms(x, eps) * weight.to(x.dtype))    # not one plus
    without("embed.norm")
    if kind == "attention":
        size = config["layers"][0]["mixer"]["mask"]["size"]
        with_patch("same_chunk", lambda T_, _: (j <= i) & (i - j < size))                                    # a sliding window
        with_patch("same_chunk", lambda T_, _: (j <= i) & ((i + 1) // size == (j + 1) // size))              # chunks from another origin
        with_patch("softmax_with_one", lambda s, seen: torch.softmax(s.masked_fill(~seen, float("-inf")), -1))    # no sink
        bucket = plain_bimolix.distance_bucket
        with_patch("distance_bucket", lambda n, rows, reach: bucket(n + 1, rows, reach))
        with_patch("distance_bucket", lambda n, rows, reach: min(n, rows - 1))                               # no logarithm
        with_patch("distance_bias", lambda T_, table, reach: table.new_zeros(table.shape[1], T_, T_))
        without("mix.q.b")
        without("mix.k.b")
        without("mix.k.norm", value=1.0)
        without("mix.g")                                                                                     # gates of a half
        without("correction")
        without("shared.sg")
        choice = plain_bimolix.router_choice
        with_patch("router_choice", lambda c, top, groups, keep: choice_by_best(c, top, groups, keep))       # groups by their best
        norm = plain_bimolix.by_rms
        values = {}

        def normed_values(h, w, prefix, mixer, eps):                                                          # values after the norm
            with monkeypatch.context() as patch:
                real = plain_bimolix.lin

                def lin(weight, x, bias=None):
                    y = real(weight, x, bias)
                    if weight is w[prefix + "k"]:
                        G, d = int(mixer["kv_heads"]), int(mixer["dim"])
                        y = (norm(y.reshape(-1, G, d), eps) * w[prefix + "k.norm"].to(y.dtype)).reshape(y.shape)
                    return y

                patch.setattr(plain_bimolix, "lin", lin)
                return values["attention"](h, w, prefix, mixer, eps)

        values["attention"] = plain_bimolix.attention
        with monkeypatch.context() as patch:
            patch.setitem(plain_bimolix.MIXERS, "attention", normed_values)
            found.append(plain(config, tensors, tokens))
    else:
        with_patch("rotate", lambda x, dims, base, first=0: x)
        with_patch("rotate", lambda x, dims, base, first=0: torch.cat([neighbours(x[..., :dims], dims, base), x[..., dims:]], -1))
        rms = plain_bimolix.by_rms
        with_patch("by_rms", lambda x, eps: rms(x.reshape(x.shape[0], -1), eps).reshape(x.shape))            # over all heads together
        with_patch("silu", lambda z: torch.sigmoid(z))
        without("mix.g")
    return found


def choice_by_best(choice, top, groups, keep):
    per = choice.shape[0] // groups
    kept = torch.topk(choice.reshape(groups, per).amax(-1), keep).indices
    open_ = torch.full_like(choice, float("-inf")).reshape(groups, per)
    open_[kept] = choice.reshape(groups, per)[kept]
    return torch.topk(open_.reshape(-1), top).indices


def neighbours(x, dims, base):
    """Pairs (2i, 2i + 1) instead of (i, i + dims/2)."""
    order = torch.cat([torch.arange(0, dims, 2), torch.arange(1, dims, 2)])
    half = dims // 2
    angle = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * (float(base) ** (-2.0 * torch.arange(half, dtype=torch.float64) / dims))
    cos, sin = torch.cos(angle)[:, None].to(x.dtype), torch.sin(angle)[:, None].to(x.dtype)
    u, v = x[..., 0::2], x[..., 1::2]
    out = torch.empty_like(x)
    out[..., order] = torch.cat([u * cos - v * sin, v * cos + u * sin], -1)
    return out


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["attention", "retention"])
def test_one_layer_alone(kind, dtype, monkeypatch, record_property):
    """A model of one layer, whole, in portions and decoded over three pages and chunks, against the plain model and
    against plain models with one constant or rule changed: the engine's logits must lie nearer to the right one."""
    config = configs.single(ONE_ATTENTION if kind == "attention" else ONE_RETENTION)
    engine, tensors = make(config, dtype, seed=11, sharp=1.5, logits=4.0)
    tokens = prompt(config, 220, 21)
    want = plain(config, tensors, tokens)
    pick = lambda value: value[dtype == "bfloat16"] if isinstance(value, tuple) else value
    others = [plain(changed(config, path, pick(value)), tensors, tokens) for path, value in OTHERS[kind]]
    others += other_rules(monkeypatch, config, tensors, tokens, kind)
    for what, sizes in (("whole", [220]), ("in portions", [61, 2, 3, 64, 1, 30, 59]), ("decoded", [50] + [1] * 170)):
        got = in_steps(engine, tokens, sizes)
        close(got, follow(engine, 0, dtype, config, tensors, tokens, want), dtype, record_property, what)
        nearer(got, follow(engine, 0, dtype, config, tensors, tokens, want), others, what, rows=slice(68, 220))


def standing_out(width, chunk, edge_bias=-9.0, others=None):
    """(config, tensors, special, asking): a model of one attention layer without distance biases to speak of whose scores lie
    far below the sink's except that of `special`, the only token with anything in channel 7, for tokens that ask for it."""
    one = configs.layer(configs.attention(2, 1, width, 4.0 / width ** 0.5, 900, chunk=chunk))
    config = configs.single(one, width=48)
    tensors = configs.tensors(config, 3, logits=3.0)
    special, asking = 5, 9
    table = tensors["embed"].float() * 0.7
    table[:, 7] = 0.0
    table[special] = 0.0
    table[special, 7] = 6.0
    table[asking, 7] = 3.0
    tensors["embed"] = table.bfloat16()
    for name, heads in (("q", 2), ("k", 1)):
        matrix = 0.05 * tensors[f"l0.mix.{name}"].float()
        matrix[::width, 7] = 2.0                          # the first entry of each head reads channel 7
        tensors[f"l0.mix.{name}"] = matrix.bfloat16()
        tensors[f"l0.mix.{name}.b"] = 0.05 * tensors[f"l0.mix.{name}.b"]
        tensors[f"l0.mix.{name}.norm"] = torch.full_like(tensors[f"l0.mix.{name}.norm"], 1.5)
    tensors["l0.mix.rel"] = torch.full_like(tensors["l0.mix.rel"], edge_bias)
    return config, tensors, special, asking


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("chunk,width", [(40, 16), (64, 64), (130, 64), (150, 24), (128, 48), (200, 128), (1, 16)])
def test_a_key_that_stands_out_at_a_chunks_edge(dtype, chunk, width, record_property):
    """Almost every weight is near zero (a large negative number at every distance) except that of a key whose token also has
    the query's direction: the same special token stands first in a chunk, last in the chunk before it, and is asked for by
    rows just behind and by the chunk's last row, in a prompt, in portions and decoded. Against plain models whose chunks
    are one position shorter or longer."""
    config, tensors, special, asking = standing_out(width, chunk)
    engine, _ = make(config, dtype, tensors=tensors)
    tokens = [t if t not in (special, asking) else 11 for t in prompt(config, 3 * chunk + 20 if chunk > 1 else 70, 4)]
    edge = 2 * chunk
    asked = [edge - 1, edge, edge + 1, min(len(tokens) - 1, edge + chunk - 1)]
    wrong = [lambda t, size=size: plain(changed(config, MIX + ("mask", "size"), size), tensors, t)
             for size in ([chunk - 1, chunk + 1] if chunk > 1 else [2])]
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


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width", [64, 48, 10])
def test_a_distance_that_stands_out(dtype, width, record_property):
    """Every bucket's number is far below zero but one's: a query sees little but the keys at the bucket's distances, its first
    and its last among them. Against plain models whose buckets begin one position earlier or later; buckets of one distance,
    of many and the last one."""
    one = configs.layer(configs.attention(4, 2, width, 0.2, 200, chunk=260))
    config = configs.single(one, width=64)
    tensors = configs.tensors(config, 3, logits=3.0, bias=0.3)
    tokens = prompt(config, 330, 4)
    bucket = plain_bimolix.distance_bucket
    for chosen in (0, 3, 15, 16, 24, 31):
        rel = torch.full((32, 4), -12.0)
        rel[chosen] = 4.0
        tensors["l0.mix.rel"] = rel.bfloat16()
        engine, _ = make(config, dtype, tensors=tensors)
        want = plain(config, tensors, tokens)
        others = []
        for shift in (-1, 1):
            with pytest.MonkeyPatch.context() as patch:
                patch.setattr(plain_bimolix, "distance_bucket", lambda n, rows, reach: bucket(max(0, n + shift), rows, reach))
                others.append(plain(config, tensors, tokens))
        others = [other for other in others if float((other - want).abs().max()) > 0.05 * float(want.abs().max())]
        assert others, "the bucket's edges do not show"
        for what, sizes in (("whole", [330]), ("portions", [100, 2, 64, 131, 33]), ("decoded", [290] + [1] * 40)):
            got = in_steps(engine, tokens, sizes)
            close(got, want, dtype, record_property, f"{what}, bucket {chosen}")
            nearer(got, want, others, (what, chosen))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("mixer", ["retention", "attention"])
def test_far_tokens_reach_the_last_rows(dtype, mixer, record_property):
    """600 tokens: the state of a slowly decaying head (or attention without chunks) carries the first forty tokens to the
    last rows; with quickly decaying heads or chunks of 150 nothing of them is left. Whole, in portions and decoded."""
    for far in (True, False):
        if mixer == "retention":
            one = configs.layer(configs.retention(2, 16, 16, (0.999, 1.0) if far else (0.3, 0.5)))
        else:
            one = configs.layer(configs.attention(2, 1, 16, 0.6, 500, chunk=None if far else 150))
        config = configs.single(one)
        engine, tensors = make(config, dtype, seed=13, sharp=2.0)
        tokens = prompt(config, 600, 3)
        other = prompt(config, 40, 4) + tokens[40:]
        want, moved = plain(config, tensors, tokens), plain(config, tensors, other)
        shift = float((want[560:] - moved[560:]).abs().max()) / float(want.abs().max())
        record_property("what the first forty tokens move the last rows by", shift)
        assert shift > 0.02 if far else shift < 1e-12
        for sequence, expected in ((tokens, want), (other, moved)):
            close(in_steps(engine, sequence, [600])[560:], expected[560:], dtype, record_property, "whole")
            close(in_steps(engine, sequence, [333, 2, 265])[560:], expected[560:], dtype, record_property, "in portions")
            close(decoded(engine, sequence, 400)[560:], expected[560:], dtype, record_property, "decoded")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("one", [ONE_ATTENTION, ONE_RETENTION])
def test_a_used_slot_is_as_good_as_a_new_one(one, dtype):
    config = configs.single(one)
    engine, tensors = make(config, dtype, seed=5)
    slot = engine.acquire()
    run(engine, slot, prompt(config, 90, 1))
    engine.release(slot)
    for length in (1, 2, 3, 5, 40):
        tokens = prompt(config, length, 30 + length)
        assert engine.acquire() == slot
        got = run(engine, slot, tokens)
        engine.release(slot)
        want = plain(config, tensors, tokens)
        close(got, follow(engine, slot, dtype, config, tensors, tokens, want), dtype, what=f"{length} tokens")
        got = decoded(engine, tokens, 1)
        close(got, follow(engine, slot, dtype, config, tensors, tokens, want), dtype, what=f"{length} tokens decoded")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layers_with_shared_tensors_keep_their_own_cache(dtype, record_property):
    """The same layer three times in a row, of both mixers: nothing of one run's cache or state reaches another's."""
    for mixer in (configs.retention(2, 16, 16, (0.9, 0.99)), configs.attention(2, 1, 16, 0.3, 40, chunk=50)):
        first = [configs.layer(mixer, configs.dense(40))]
        config = configs.model(67, 48, 1e-5, first + [configs.again(first, 0), configs.again(first, 0)], positions=400)
        engine, tensors = make(config, dtype, seed=5)
        tokens = prompt(config, 130, 7)
        want = plain(config, tensors, tokens)
        once = plain(dict(config, layers=config["layers"][:1]), tensors, tokens)
        for what, sizes in (("whole", [130]), ("portions", [40, 2, 88]), ("decoded", [60] + [1] * 70)):
            got = in_steps(engine, tokens, sizes)
            close(got, want, dtype, record_property, what)
            nearer(got, want, [once], what)


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
    config = configs.model(101, 128, 1e-5, [
        configs.layer(configs.retention(2, 64, 64, (0.9, 0.9995)), configs.dense(64)),
        configs.layer(configs.attention(4, 2, 64, 0.15, 200, chunk=300)),
        configs.layer(configs.attention(2, 2, 16, 0.3, 700), configs.dense(64)),
        configs.layer(configs.retention(3, 16, 16))], positions=1600)
    engine, tensors = make(config, dtype, seed=8, max_tokens=4096)
    tokens = prompt(config, 1400, 2)
    want = plain(config, tensors, tokens)
    close(in_steps(engine, tokens, [1400]), want, dtype, record_property, "whole")
    close(decoded(engine, tokens, 1100), want, dtype, record_property, "decoded")


def test_which_kernels_run(record_property):
    """The bfloat16 engine takes the tensor-core attention kernels (tcgen05 for prompts at head widths 64 and 128, mma.sync
    else, and in decoding) with the norm, the cache write and the gate inside where a token is decoded, chunked retention for
    prompts and one kernel a retention layer in decoding; the 32-bit engine takes the general kernels and the 32-bit product
    only."""
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
    assert names.count("retention[chunks]") == 4 and names.count("rotate_heads") == 1 == names.count("scalar_recurrence")
    assert names.count("head_norm_gate") == 1 and "attention" not in names and "sigmoid_gate" not in names
    assert names.count("gemm_bounded_gate[tcgen05, groups]") == 3
    with ops.record_launches() as names:
        last = run(engine, slot, tokens[299:])
    record_property("decode kernels", sorted(set(names)))
    assert sum(name.startswith("attention_decode") for name in names) == 5 and "sigmoid_gate" not in names
    assert names.count("rope_store") == 1                            # twelve heads a key/value head: the norm in a kernel of its own
    assert names.count("retention[one token]") == 5 and names.count("gemm_bounded_gate[skinny]") == 2
    engine.release(slot)
    close(last, follow(engine, slot, "bfloat16", config, tensors, tokens, want)[299:], "bfloat16", record_property, "decoded", slack=2.0)
    engine32, _ = make(config, "float32", seed=3)
    slot = engine32.acquire()
    with ops.record_launches() as names:
        run(engine32, slot, tokens)
    assert "library_mm" not in names and "retention[chunks]" not in names
    assert not any("tensor" in name or "tcgen05" in name or "skinny" in name or "mma" in name for name in names)


# ------------------------------------------------------------------ generation, the command line, the trace runner
def teacher_forced(config, tensors, request, tokens, bound, engine=None):
    """(close calls, misses): tokens whose two best logits lie closer than the bound (either may be taken), and
    tokens that are not the plain model's choice although it was clear. With `engine` the plain model takes its choice of
    experts at close calls (the sequence is decoded once more for them)."""
    choices = None
    if engine is not None:
        slot = engine.acquire()
        run(engine, slot, request, want=[])
        for token in tokens:
            run(engine, slot, [token])
        engine.release(slot)
        choices = engine.choices[slot] or None
    logits = plain(config, tensors, list(request) + list(tokens), choices)[len(request) - 1:-1].numpy()
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
    counts = [teacher_forced(config, tensors, r, t, GREEDY[dtype], engine if dtype == "bfloat16" else None)
              for r, t in zip(requests, found)]
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
    """bin/trace_run on a Bimolix folder: three unequal requests start together (one of a single token), are decoded
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
