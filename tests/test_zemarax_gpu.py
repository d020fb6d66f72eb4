"""The Zemarax decoder in the engine against the plain implementation (plain_zemarax.py): each mechanism's kernel
alone, then whole models under every kind of schedule."""

from __future__ import annotations

import json

import pytest
import torch

import harness
import plain_zemarax as plain
import zemarax_tiny as zt

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def _ops():
    from pulsarlm_b200.kernels import ops

    ops.require_device()
    return ops


def _i32(values):
    return torch.tensor(values, dtype=torch.int32, device=DEV)


def _bar(dtype) -> float:
    return 1e-5 if dtype == torch.float32 else 1e-2


def _paged(lengths, page, gen):
    """A block table over pages handed out in a scrambled order."""
    n_pages = sum(-(-n // page) for n in lengths) + 2
    order = torch.randperm(n_pages, generator=gen).tolist()
    table = torch.full((len(lengths), max(-(-n // page) for n in lengths)), -1, dtype=torch.int32)
    for e, n in enumerate(lengths):
        for j in range(-(-n // page)):
            table[e, j] = order.pop()
    return n_pages, table


# --------------------------------------------------------------------------- embedding

@pytest.mark.parametrize("width", [24, 30])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_scaled_pair_embedding_with_positions(width, dtype):
    """Portions and single tokens of three requests; the scale touches the table's row only, positions go on where the
    last step stopped; a position past the table's end raises the status word."""
    ops = _ops()
    gen = torch.Generator().manual_seed(5)
    vocab, buckets, positions, scale = 50, 13, 20, 4.0
    cfg = {"embedding": {"scale": scale, "bigram": {"buckets": buckets, "mul_prev": 7, "mul_cur": 3}}}
    table, pairs, places = (torch.randn(n, width, generator=gen).to(dtype) for n in (vocab, buckets + 1, positions))
    state = torch.full((5,), 49, dtype=torch.int32, device=DEV)   # (what an earlier owner of a slot left behind)
    seqs = {r: torch.randint(0, vocab, (n,), generator=gen).tolist() for r, n in {0: 9, 1: 6, 2: 4}.items()}
    slot_of = {0: 2, 1: 0, 2: 3}
    want = {r: plain.embedding(s, table.double(), pairs.double(), places.double(), cfg) for r, s in seqs.items()}
    fed = {r: 0 for r in seqs}
    status = torch.zeros(1, dtype=torch.int32, device=DEV)

    def run(tokens, pos, entry, slots, single):
        out = torch.empty(len(tokens), width, dtype=torch.float32, device=DEV)
        ops.pair_embed(table.to(DEV), pairs.to(DEV), _i32(tokens), _i32(pos), _i32(entry), _i32(slots), state, out, 7, 3,
                       single, status, scale, places.to(DEV))
        return out.cpu()

    for step in ([(0, 4), (1, 2)], [(2, 1), (0, 1), (1, 3)], [(0, 1), (1, 1), (2, 1)], [(2, 2), (0, 3)]):
        tokens, pos, entry, slots, rows = [], [], [], [], []
        for e, (r, n) in enumerate(step):
            tokens += seqs[r][fed[r]: fed[r] + n]
            pos += list(range(fed[r], fed[r] + n))
            entry += [e] * n
            slots.append(slot_of[r])
            rows.append((r, fed[r], n))
            fed[r] += n
        out, at = run(tokens, pos, entry, slots, all(n == 1 for _, n in step)), 0
        for r, start, n in rows:
            assert plain.relative_error_of(out[at: at + n], want[r][start: start + n]) < 1e-6, (step, r)
            at += n
    assert int(status.item()) == 0
    run([1], [positions], [0], [1], True)
    assert int(status.item()) == 1


# --------------------------------------------------------------------------- attention

def _attention_case(gen, lengths, heads, kv, dim, page, dtype, spikes, queries):
    """Paged keys and values, queries for chosen (request, position) pairs; `spikes(position)` lists key positions that are
    lined up with the query's head 0 (and, smaller, with the other heads of its kv head)."""
    n_pages, table = _paged(lengths, page, gen)
    keys = [torch.randn(n, kv, dim, generator=gen).to(dtype) for n in lengths]
    values = [torch.randn(n, kv, dim, generator=gen).to(dtype) for n in lengths]
    q_full = [torch.randn(n, heads, dim, generator=gen).to(dtype) for n in lengths]
    direction = torch.randn(dim, generator=gen)
    direction = direction / direction.norm()
    for e, p in queries:
        q_full[e][p, 0] = (6.0 * direction).to(dtype)   # (one direction for every query: spikes at fixed places serve all)
        for j in spikes(p):
            if 0 <= j < lengths[e]:
                keys[e][j, 0] = (7.0 * direction).to(dtype)
    pools = torch.zeros(n_pages, 2, kv, page, dim, dtype=dtype, device=DEV)
    for e, n in enumerate(lengths):
        for j in range(n):
            pools[table[e, j // page], 0, :, j % page] = keys[e][j].to(DEV)
            pools[table[e, j // page], 1, :, j % page] = values[e][j].to(DEV)
    return table, keys, values, q_full, pools


def _wanted(keys, values, q_full, scale, window, keep, sink, queries):
    full = [plain.sink_attention(q_full[e].double(), keys[e].double(), values[e].double(), scale,
                                 plain.in_reach(keys[e].shape[0], window, keep), sink) for e in range(len(keys))]
    return torch.stack([full[e][p] for e, p in queries])


def _holes(table, lengths, page, window, keep, queries_from):
    """The block table as the cache keeps it: pages neither kept nor in any remaining query's window are -1."""
    table = table.clone()
    if window is None:
        return table
    for e, n in enumerate(lengths):
        first = max(0, queries_from[e] - window + 1) // page
        for j in range(-(-keep // page), min(first, table.shape[1])):
            table[e, j] = -1
    return table


REACH = [(None, 0), (21, 3), (24, 16), (24, 17), (37, 5), (16, 48), (7, 40), (1, 1), (64, 64), (70, 65), (33, 0)]


def _spike_sets(window, keep):
    """No spike; the window's oldest key; the first one outside it; the last kept key; the first one not kept."""
    out = {"none": lambda p: []}
    if window is not None:
        out["window_in"] = lambda p: [p - window + 1]
        out["window_out"] = lambda p: [p - window]
        if keep:
            out["kept"] = lambda p: [keep - 1]
        out["not_kept"] = lambda p: [keep]
    return out


@pytest.mark.parametrize("window,keep", REACH)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_kept_first_keys_on_the_cuda_core_kernel(window, keep, dtype):
    ops = _ops()
    heads, kv, dim, page, scale = 6, 2, 16, 8, 0.3
    lengths = [170, 33, 8, 129]
    for name, spikes in _spike_sets(window, keep).items():
        gen = torch.Generator().manual_seed(11)
        queries = [(e, p) for e, n in enumerate(lengths) for p in sorted({0, 1, n // 2, n - 2, n - 1})]
        if name != "none":
            queries = [(e, n - 1) for e, n in enumerate(lengths)]   # (a spike is one query's edge and another's middle)
        table, keys, values, q_full, pools = _attention_case(gen, lengths, heads, kv, dim, page, dtype, spikes, queries)
        sink = torch.randn(heads, generator=gen)
        want = _wanted(keys, values, q_full, scale, window, keep, sink, queries)
        if name != "none":
            table = _holes(table, lengths, page, window, keep, [n - 1 for n in lengths])
        q = torch.stack([q_full[e][p] for e, p in queries]).to(DEV)
        out = torch.empty_like(q)
        status = torch.zeros(1, dtype=torch.int32, device=DEV)
        ops.attention_simt(q, pools[:, 0], pools[:, 1], table.to(DEV), _i32([p for _, p in queries]),
                           _i32([e for e, _ in queries]), out, page, window, scale, status, sinks=sink.to(DEV), keep_first=keep)
        assert int(status.item()) == 0 and plain.relative_error_of(out.cpu(), want) < _bar(dtype), name


@pytest.mark.parametrize("dim,heads,kv", [(32, 6, 2), (64, 8, 4), (64, 3, 3), (80, 6, 3), (128, 8, 1), (128, 3, 1)])
@pytest.mark.parametrize("window,keep", REACH)
def test_kept_first_keys_and_sinks_on_the_tensor_core_kernels(dim, heads, kv, window, keep):
    """bfloat16 single tokens (any number of key shares) and prompt rows (mma.sync, and tcgen05 where it takes the
    shape, with and without split keys), with pages behind the window taken away."""
    ops = _ops()
    page, scale, dtype = 16, 0.25, torch.bfloat16
    lengths = [300, 33, 16, 129]
    for name, spikes in _spike_sets(window, keep).items():
        gen = torch.Generator().manual_seed(21)
        queries = [(e, n - 1) for e, n in enumerate(lengths)]
        table, keys, values, q_full, pools = _attention_case(gen, lengths, heads, kv, dim, page, dtype, spikes, queries)
        sink = torch.randn(heads, generator=gen)
        want = _wanted(keys, values, q_full, scale, window, keep, sink, queries)
        holed = _holes(table, lengths, page, window, keep, [n - 1 for n in lengths]).to(DEV)
        q = torch.stack([q_full[e][p] for e, p in queries]).to(DEV)
        pos, entry = _i32([p for _, p in queries]), _i32([e for e, _ in queries])
        status = torch.zeros(1, dtype=torch.int32, device=DEV)
        for splits in (1, 2, 5):
            scratch = torch.empty(ops.attention_decode_scratch_floats(len(queries), heads, dim, splits), dtype=torch.float32,
                                  device=DEV) if splits > 1 else None
            out = torch.empty_like(q)
            ops.attention_decode(q, pools[:, 0], pools[:, 1], holed, pos, entry, out, page, window, scale, splits, scratch,
                                 status, extras=ops.attention_extras(q, sink.to(DEV), None, False, 0.0, None, None, keep))
            assert plain.relative_error_of(out.cpu(), want) < 1e-2, ("single tokens", name, splits)
        assert int(status.item()) == 0, name
    # prompt rows: portions of the requests as tiles; every query of a portion sees its own window
    spans = [(0, 170, 300), (3, 0, 129), (1, 32, 33), (2, 0, 16)]
    for name, spikes in _spike_sets(window, keep).items():
        gen = torch.Generator().manual_seed(22)
        queries = [(e, p) for e, lo, hi in spans for p in range(lo, hi)]
        marked = queries if name == "none" else [(0, 299), (3, 128), (1, 32), (2, 15)]
        table, keys, values, q_full, pools = _attention_case(gen, lengths, heads, kv, dim, page, dtype, spikes, marked)
        sink = torch.randn(heads, generator=gen)
        want = _wanted(keys, values, q_full, scale, window, keep, sink, queries)
        holed = _holes(table, lengths, page, window, keep, [170, 32, 0, 0]).to(DEV)
        q = torch.stack([q_full[e][p] for e, p in queries]).to(DEV)
        group = heads // kv

        def tiles_of(rows):
            tiles, at = [], 0
            for e, lo, hi in spans:
                tiles += [(at + r, min(rows, hi - lo - r), lo + r, e) for r in range(0, hi - lo, rows)]
                at += hi - lo
            return _i32(tiles)

        status = torch.zeros(1, dtype=torch.int32, device=DEV)
        out = torch.empty_like(q)
        ops.attention_prefill(q, pools[:, 0], pools[:, 1], holed, tiles_of(ops.attention_prefill_tile_rows()), out, page, window,
                              scale, status, extras=ops.attention_extras(q, sink.to(DEV), None, False, 0.0, None, None, keep))
        assert int(status.item()) == 0 and plain.relative_error_of(out.cpu(), want) < 1e-2, ("prompt rows", name)
        if ops.attention_prefill_tcgen05_supports(q, pools[:, 0], page):
            for rows in sorted({ops.attention_prefill_tile_rows(), ops.attention_prefill_tcgen05_tile_rows(group)}):
                for splits in (1, 2, 3):
                    scratch = torch.empty(ops.attention_prefill_scratch_floats(q.shape[0], heads, dim, splits),
                                          dtype=torch.float32, device=DEV) if splits > 1 else None
                    out = torch.empty_like(q)
                    ops.attention_prefill_tcgen05(q, pools[:, 0], pools[:, 1], holed, tiles_of(rows), out, page, window, scale,
                                                  status, splits, scratch, sinks=sink.to(DEV), keep_first=keep)
                    assert int(status.item()) == 0
                    assert plain.relative_error_of(out.cpu(), want) < 1e-2, ("prompt rows on tcgen05", name, rows, splits)


@pytest.mark.parametrize("rank,heads", [(64, 4), (128, 16), (64, 3), (128, 5), (64, 1)])
@pytest.mark.parametrize("spike", [None, 0, 15, 100])
def test_rows_that_are_keys_and_values_on_tcgen05(rank, heads, spike):
    """Prompt rows over one pool (a cached latent), a sink per head, one key at a chosen place that stands out."""
    ops = _ops()
    page, scale, dtype, lengths = 16, 0.25, torch.bfloat16, [300, 33, 16, 129]
    spans = [(0, 170, 300), (3, 0, 129), (1, 32, 33), (2, 0, 16)]
    gen = torch.Generator().manual_seed(rank + heads)
    queries = [(e, p) for e, lo, hi in spans for p in range(lo, hi)]
    table, keys, _, q_full, pools = _attention_case(gen, lengths, heads, 1, rank, page, dtype,
                                                    lambda p: [] if spike is None else [spike], [(0, 299), (3, 128)])
    sink = torch.randn(heads, generator=gen)
    want = _wanted(keys, keys, q_full, scale, None, 0, sink, queries)
    q, pool = torch.stack([q_full[e][p] for e, p in queries]).to(DEV), pools[:, 0].contiguous()
    assert ops.attention_prefill_tcgen05_supports_shared(rank, heads, pool, page)
    tiles, at, rows = [], 0, ops.attention_prefill_tcgen05_tile_rows(heads)
    for e, lo, hi in spans:
        tiles += [(at + r, min(rows, hi - lo - r), lo + r, e) for r in range(0, hi - lo, rows)]
        at += hi - lo
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    for with_sink in (True, False):
        wanted = want if with_sink else _wanted(keys, keys, q_full, scale, None, 0, None, queries)
        for splits in (1, 3):
            scratch = torch.empty(ops.attention_prefill_scratch_floats(q.shape[0], heads, rank, splits), dtype=torch.float32,
                                  device=DEV) if splits > 1 else None
            out = torch.empty_like(q)
            ops.attention_prefill_tcgen05(q, pool, pool, table.to(DEV), _i32(tiles), out, page, None, scale, status, splits,
                                          scratch, heads % 2 == 1, sinks=sink.to(DEV) if with_sink else None)
            assert int(status.item()) == 0 and plain.relative_error_of(out.cpu(), wanted) < 1e-2, (with_sink, splits)


# --------------------------------------------------------------------------- matrix memory

def _memory_case(gen, steps, heads, dim, vdim, hidden, dtype, forget=3.0):
    """h and the projections' weights of one sequence; f's bias spreads memories from short to long."""
    w = {n: torch.randn(r, hidden, generator=gen) / hidden ** 0.5 for n, r in
         (("q", heads * dim), ("k", heads * dim), ("v", heads * vdim), ("g", heads * vdim), ("i", heads), ("f", heads))}
    w = {n: x.to(dtype) for n, x in w.items()}
    w["i.b"], w["f.b"] = torch.randn(heads, generator=gen), forget + 2.0 * torch.randn(heads, generator=gen)
    w["norm"] = 1.0 + 0.2 * torch.randn(heads * vdim, generator=gen)
    w["o"] = torch.eye(heads * vdim).to(dtype)
    return torch.randn(steps, hidden, generator=gen).to(dtype), w


def _memory_part(w, heads, dim, vdim, hidden, cap, eps, dtype, slots):
    from pulsarlm_b200.cache.manager import StateBinding
    from pulsarlm_b200.parts.registry import BuildContext, build_part
    from pulsarlm_b200.parts.spec import PartSpec

    spec = PartSpec("matrix_memory", {"hidden_size": hidden, "n_heads": heads, "head_dim": dim, "value_dim": vdim,
                                      "gate_cap": cap, "eps": eps},
                    {**{n: n for n in ("q", "k", "v", "g", "i", "f", "norm", "o")}, "i_bias": "i.b", "f_bias": "f.b"})
    part = build_part("mixer", spec, BuildContext(dtype, torch.device(DEV)))
    part.load({n: x.to(DEV) for n, x in w.items()})
    need = part.cache_need()
    # (slots start at zero as the cache manager zeroes them; the others hold another request's state)
    part.bind_cache(StateBinding(torch.zeros((slots, *need.shape), dtype=torch.float32, device=DEV)))
    return part


def _memory_steps(part, sequences, schedule, slot_of):
    """Feeds {request: h [T, H]} by a schedule of steps [(request, rows), ...]; returns {request: outputs}."""
    from pulsarlm_b200.models.model import HostStep, StepBatch

    fed = {r: 0 for r in sequences}
    got = {r: [] for r in sequences}
    for step in schedule:
        step = sorted(step, key=lambda x: x[1] != 1)   # (entries of one token lead)
        lens = [n for _, n in step]
        firsts = [sum(lens[:i]) for i in range(len(lens))]
        h = torch.cat([sequences[r][fed[r]: fed[r] + n] for r, n in step]).to(DEV)
        n_decode = sum(1 for n in lens if n == 1)
        host = HostStep(len(step), h.shape[0], n_decode, lens, [fed[r] + n for r, n in step], firsts, 16)
        plan = {k: torch.from_numpy(v).to(DEV) if v is not None else None for k, v in part.plan_step(host).items()}
        pos = torch.cat([torch.arange(fed[r], fed[r] + n) for r, n in step]).int().to(DEV)
        entry = torch.cat([torch.full((n,), e) for e, n in enumerate(lens)]).int().to(DEV)
        batch = StepBatch(pos, pos, entry, {}, _i32([slot_of[r] for r, _ in step]), None,
                          torch.zeros(1, dtype=torch.int32, device=DEV), h.shape[0], len(step), n_decode, lens,
                          plans={part.plan_key(): plan})
        out = part.forward(h, batch).cpu()
        for (r, n), at in zip(step, firsts):
            got[r].append(out[at: at + n])
            fed[r] += n
    assert all(fed[r] == sequences[r].shape[0] for r in sequences)
    return {r: torch.cat(x) for r, x in got.items()}


SHAPES = [(6, 32, 64), (3, 16, 24), (2, 64, 128), (5, 6, 10), (2, 48, 80), (1, 128, 64), (2, 256, 40), (3, 8, 4), (2, 20, 200),
          (1, 96, 512), (2, 40, 1)]


@pytest.mark.parametrize("heads,dim,vdim", SHAPES)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_matrix_memory_in_portions_and_token_by_token(heads, dim, vdim, dtype):
    """Whole, in portions that begin and end anywhere in a chunk, token by token, and three requests side by side
    (portions beside single tokens); a slot taken again starts from zero; float32 bits do not depend on the cut."""
    _ops()
    hidden, cap, eps, steps = 40, 6.0, 1e-5, 150
    gen = torch.Generator().manual_seed(heads * 1000 + dim + vdim)
    h, w = _memory_case(gen, steps, heads, dim, vdim, hidden, dtype)
    m = {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}

    def plain_out(x):
        return plain.matrix_memory_mixer(x.double(), {n: t.double() for n, t in w.items()}, m, eps,
                                         lambda t: t.to(dtype).double())

    part = _memory_part(w, heads, dim, vdim, hidden, cap, eps, dtype, 5)
    # (the norm of a head of one column is x / sqrt(x^2 + eps): near zero it multiplies an error by up to 1 / sqrt(eps))
    want, bar = plain_out(h), (2e-5 if vdim > 1 else 5e-4) if dtype == torch.float32 else 2e-2

    def alone(cuts):
        part.states[2].zero_()
        part.states[[0, 1, 3, 4]] = 9.0
        return _memory_steps(part, {"a": h}, [[("a", n)] for n in cuts], {"a": 2})["a"]

    whole = alone([steps])
    assert plain.relative_error_of(whole, want) < bar
    for cuts in ([64, 86], [1, 2, 61, 63, 1, 1, 2, 19], [70, 2, 2, 2, 65, 9], [128, 22], [2] * 75):
        got = alone(cuts)
        assert plain.relative_error_of(got, want) < bar, cuts
        assert dtype == torch.bfloat16 or torch.equal(got, whole), cuts
    single = alone([1] * steps)
    assert plain.relative_error_of(single, want) < bar
    assert dtype == torch.bfloat16 or torch.equal(single, whole)
    assert float((part.states[[0, 1, 3, 4]] - 9.0).abs().max()) == 0.0
    sequences = {"a": h, "b": torch.randn(67, hidden, generator=gen).to(dtype), "c": torch.randn(131, hidden, generator=gen).to(dtype)}
    part.states.zero_()
    schedule = [[("a", 20), ("b", 1)], [("a", 1), ("b", 64), ("c", 66)], [("a", 128), ("c", 1), ("b", 1)],
                [("b", 1), ("c", 63)], [("c", 1), ("a", 1)]]
    got = _memory_steps(part, sequences, schedule, {"a": 3, "b": 0, "c": 4})
    for r, x in sequences.items():
        assert plain.relative_error_of(got[r], plain_out(x)) < bar, r


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_matrix_memory_keeps_and_forgets(dtype):
    """Gates at their extremes: forget gates so open that the first token still matters 2,000 tokens on, so closed that only
    the last token does, input gates at the cap's both ends (the stabiliser follows them up and down)."""
    _ops()
    heads, dim, vdim, hidden, cap, eps = 4, 32, 32, 24, 15.0, 1e-5
    gen = torch.Generator().manual_seed(3)
    h, w = _memory_case(gen, 2000, heads, dim, vdim, hidden, dtype)
    w["f.b"] = torch.tensor([14.0, -40.0, 9.0, 2.0])
    w["i.b"] = torch.tensor([0.0, 0.0, 30.0, -30.0])
    w["i"] = w["i"] * 8
    w["i"][0] = 0.0   # (every token enters head 0 alike)
    m = {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}
    plain_w = {n: t.double() for n, t in w.items()}

    def plain_out(x):
        return plain.matrix_memory_mixer(x.double(), plain_w, m, eps, lambda t: t.to(dtype).double())

    want = plain_out(h)
    part = _memory_part(w, heads, dim, vdim, hidden, cap, eps, dtype, 2)
    got = _memory_steps(part, {"a": h}, [[("a", 700)], [("a", 1290)]] + [[("a", 1)]] * 10, {"a": 1})["a"]
    assert plain.relative_error_of(got, want) < (1e-4 if dtype == torch.float32 else 2e-2)
    # the first token matters to the end where the gate is open
    other = h.clone()
    other[0] = torch.randn(hidden, generator=gen).to(dtype)
    part.states.zero_()
    moved = _memory_steps(part, {"a": other}, [[("a", 2000)]], {"a": 1})["a"]
    change = (moved[-1] - got[-1]).abs().view(heads, vdim).amax(1)
    wanted = (plain_out(other)[-1] - want[-1]).abs().view(heads, vdim).amax(1)
    assert float(wanted[0]) > 1e-3 and float(wanted[1]) < 1e-9
    if dtype == torch.float32:
        assert abs(float(change[0] - wanted[0])) < 0.05 * float(wanted[0])


# --------------------------------------------------------------------------- latents, router, experts

@pytest.mark.parametrize("query_rank,rank", [(128, 64), (20, 33), (512, 96), (7, 4)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_two_latents_normed_in_one_launch(query_rank, rank, dtype):
    ops = _ops()
    gen = torch.Generator().manual_seed(rank)
    lengths, page, eps = [21, 5], 8, 1e-5
    tokens = sum(lengths)
    proj = torch.randn(tokens, query_rank + rank + 4, generator=gen).to(dtype)
    wq, wk = 1.0 + 0.3 * torch.randn(query_rank, generator=gen), 1.0 + 0.3 * torch.randn(rank, generator=gen)
    n_pages, table = _paged(lengths, page, gen)
    pos = torch.cat([torch.arange(n) for n in lengths])
    entry = torch.cat([torch.full((n,), e) for e, n in enumerate(lengths)])
    dev = proj.to(DEV)
    for cached in (True, False):
        pool = torch.full((n_pages, 1, page, rank), 7.0, dtype=dtype, device=DEV)
        out = torch.empty(tokens, query_rank, dtype=dtype, device=DEV)
        ops.latent_norms(dev[:, :query_rank], wq.to(DEV), out, dev[:, query_rank: query_rank + rank] if cached else None,
                         wk.to(DEV), eps, pos.int().to(DEV), entry.int().to(DEV), table.to(DEV), pool if cached else None, page)
        assert plain.relative_error_of(out.cpu(), plain.rms(proj[:, :query_rank].double(), eps) * wq.double()) < _bar(dtype)
        want = plain.rms(proj[:, query_rank: query_rank + rank].double(), eps) * wk.double()
        if cached:
            got = torch.stack([pool[table[int(e), int(p) // page], 0, int(p) % page].cpu() for e, p in zip(entry, pos)])
            assert plain.relative_error_of(got, want) < _bar(dtype)
        else:
            assert float((pool - 7.0).abs().max()) == 0.0


@pytest.mark.parametrize("experts,top", [(8, 4), (5, 1), (6, 6), (64, 6), (3, 2)])
@pytest.mark.parametrize("tokens", [3, 300])
def test_router_with_biased_logits_and_weights_over_the_chosen(experts, top, tokens):
    """A bias that changes the choice and the weights, beside a shared expert's gate as the router's last row."""
    ops = _ops()
    gen = torch.Generator().manual_seed(experts)
    hidden = 40
    h, router = torch.randn(tokens, hidden, generator=gen), torch.randn(experts + 1, hidden, generator=gen) * 0.5
    bias = 3.0 * torch.randn(experts, generator=gen)
    ids, weights = plain.route(h.double(), router[:experts].double(), bias.double(), top)
    shared = torch.empty(tokens, dtype=torch.float32, device=DEV)
    got_ids, got_w = ops.moe_route(h.to(DEV), router.to(DEV), None, top, 1, 1, False, 1, True, shared, bias.to(DEV))
    assert torch.equal(got_ids.cpu().long(), ids)
    assert plain.relative_error_of(got_w.cpu(), weights) < 1e-5
    assert plain.relative_error_of(shared.cpu(), torch.sigmoid(h.double() @ router[experts].double())) < 1e-5


@pytest.mark.parametrize("tokens", [5, 130])
@pytest.mark.parametrize("shared", [40, None])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_routed_gelu_experts(tokens, shared, dtype):
    """The feed-forward part alone, few tokens (every pair streams its expert) and many (grouped products)."""
    from pulsarlm_b200.parts.registry import BuildContext, build_part
    from pulsarlm_b200.parts.spec import PartSpec

    _ops()
    gen = torch.Generator().manual_seed(3)
    width, ff, experts, top = 48, 24, 8, 3
    mlp = zt.routed(ff, experts, top, shared)
    w = {"router": torch.randn(experts, width, generator=gen) * 0.5, "router.b": torch.randn(experts, generator=gen)}
    for e in range(experts):
        w[f"e{e}.up"] = 2.0 * torch.randn(ff, width, generator=gen) / width ** 0.5
        w[f"e{e}.down"] = torch.randn(width, ff, generator=gen) / ff ** 0.5
    if shared:
        w["shared.up"] = 2.0 * torch.randn(shared, width, generator=gen) / width ** 0.5
        w["shared.down"] = torch.randn(width, shared, generator=gen) / shared ** 0.5
        w["shared.sg"] = torch.randn(1, width, generator=gen) / width ** 0.5
    w = {k: v.to(dtype) for k, v in w.items()}
    h = torch.randn(tokens, width, generator=gen).to(dtype)
    want = plain.routed_ff(h.double(), {k: v.double() for k, v in w.items()}, mlp, lambda t: t)
    names = {"router": "router", "logit_bias": "router.b", "expert_up": "e{e}.up", "expert_down": "e{e}.down"}
    if shared:
        names.update(shared_up="shared.up", shared_down="shared.down", shared_gate_row="shared.sg")
    part = build_part("feed_forward", PartSpec("moe", {"hidden_size": width, "expert_size": ff, "n_experts": experts, "top": top,
                                                       "shared_size": shared, "expert": "gelu"}, names),
                      BuildContext(dtype, torch.device(DEV)))
    part.load({k: v.to(DEV) for k, v in w.items()})
    assert plain.relative_error_of(part.forward(h.to(DEV), None).cpu(), want) < (1e-5 if dtype == torch.float32 else 2e-2)


@pytest.mark.parametrize("width", [64, 30])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_exact_gelu(width, dtype):
    ops = _ops()
    z = torch.linspace(-12.0, 12.0, 50 * width).view(50, width).to(dtype)
    out = torch.empty_like(z, device=DEV)
    ops.bias_act(z.to(DEV), None, out, "gelu")
    want = plain.gelu(z.double())
    assert plain.relative_error_of(out.cpu(), want) < _bar(dtype)
    # relative accuracy in the negative tail, where 1 + erf cancels
    tail = (z.double() > -5.0) & (z.double() < -2.0)
    assert float(((out.cpu().double() - want) / want)[tail].abs().max()) < (1e-5 if dtype == torch.float32 else 1e-2)


# --------------------------------------------------------------------------- whole models

def _model(key, dtype, seed=1, sharp=1.0):
    return zt.TinyZemarax(key, dtype, seed, sharp=sharp)


def _portions(tokens, cuts, request="p", want_all=True):
    assert sum(cuts) == len(tokens)
    steps, at = [], 0
    for n in cuts:
        steps.append(([(request, tokens[at: at + n], list(range(n)) if want_all else [n - 1])], []))
        at += n
    return steps


@pytest.mark.parametrize("key", ["A", "B", "C"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_prompts_and_their_first_tokens(key, dtype):
    tm = _model(key, dtype)
    runner = tm.runner(24)
    tokens = {"p": zt.random_tokens(tm.cfg, 175, 3), "q": zt.random_tokens(tm.cfg, 5, 4), "r": zt.random_tokens(tm.cfg, 1, 5)}
    got = harness.replay(runner, [([("p", tokens["p"], list(range(175)))], ["p"]),
                                  ([("q", tokens["q"], list(range(5)))], ["q"]),
                                  ([("r", tokens["r"], [0])], ["r"])])
    tm.check(tokens, got, f"{key} whole")


def test_residual_stream_after_every_layer():
    """float32: the stream after each layer of a prompt fed in two portions, against the plain implementation's, so that
    a fault is placed at its layer."""
    from pulsarlm_b200.engine.runner import StepEntry
    from pulsarlm_b200.parts.basic import settle_pending

    for key in ("A", "B", "C"):
        tm = _model(key, "float32")
        tokens = zt.random_tokens(tm.cfg, 37, 9)
        want: list = []
        plain.forward(tm.cfg, tm.plain_weights, tokens, streams=want)
        runner = tm.runner(8)
        seen: list = []
        for block in runner.model.blocks:
            def wrapped(x, delta, batch, inner=block.forward):
                x, pending = inner(x, delta, batch)
                settled = x.clone()
                settle_pending(settled, pending)
                seen.append(settled.cpu())
                return x, pending
            block.forward = wrapped
        runner.step([StepEntry("p", tokens[:20], [19])])
        runner.step([StepEntry("p", tokens[20:], [16])])
        layers = len(tm.cfg["layers"])
        for i in range(layers):
            assert plain.relative_error_of(torch.cat([seen[i], seen[layers + i]]), want[i]) < 2e-5, (key, i)


@pytest.mark.parametrize("key", ["A", "B", "C"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prefill_then_token_by_token(key, dtype):
    """A prompt in one step, then 110 tokens one by one: past every window and over page borders."""
    tm = _model(key, dtype)
    runner = tm.runner(24)
    tokens = {"p": zt.random_tokens(tm.cfg, 150, 5)}
    steps = [([("p", tokens["p"][:40], [0, 1, 39])], [])]
    steps += [([("p", [tokens["p"][i]], [0])], []) for i in range(40, 150)]
    tm.check(tokens, harness.replay(runner, steps), f"{key} decode")


@pytest.mark.parametrize("key", ["A", "B", "C"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_token_by_token_from_the_start(key, dtype):
    """The first tokens of a sequence: the pair table's last row, kept keys while they are still in the window, states
    from zero."""
    tm = _model(key, dtype)
    runner = tm.runner(8)
    tokens = {"p": zt.random_tokens(tm.cfg, 30, 6)}
    tm.check(tokens, harness.replay(runner, [([("p", [t], [0])], []) for t in tokens["p"]]), f"{key} from the start")


@pytest.mark.parametrize("key", ["A", "B", "C"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_of_many_sizes(key, dtype):
    tm = _model(key, dtype)
    runner = tm.runner(24)
    tokens = {"p": zt.random_tokens(tm.cfg, 217, 7)}
    cuts = [2, 2, 3, 1, 1, 7, 16, 2, 33, 1, 2, 17, 31, 2, 30, 65, 2]
    tm.check(tokens, harness.replay(runner, _portions(tokens["p"], cuts)), f"{key} portions")


@pytest.mark.parametrize("key", ["A", "B"])
def test_float32_bits_do_not_depend_on_the_cut(key):
    """In float32 every kernel adds in an order fixed by the token's own place: logits of a prompt fed whole and fed in
    portions are equal bit for bit."""
    tm = _model(key, "float32")
    tokens = zt.random_tokens(tm.cfg, 90, 8)
    whole = harness.replay(tm.runner(12), [([("p", tokens, list(range(90)))], [])])["p"]
    cut = harness.replay(tm.runner(12), _portions(tokens, [5, 1, 2, 40, 1, 1, 3, 37]))["p"]
    for position in range(90):
        assert torch.equal(whole[position], cut[position]), position


@pytest.mark.parametrize("key", ["A", "B", "C"])
@pytest.mark.parametrize("sharp", [3.0, 6.0])
def test_sharp_attention_shows_every_key_in_reach(key, sharp):
    """float32, scores multiplied so that each softmax rests on a few keys. Prompt portions whose cuts fall just before, at
    and just after every window's edge and past the kept tokens, then single tokens until every window has passed over
    decoded tokens, with pages of 16 and of 64."""
    tm = _model(key, "float32", seed=7, sharp=sharp)
    masks = [(entry["mixer"].get("mask") or {}) for entry in tm.cfg["layers"]]
    windows = sorted({m["size"] for m in masks if m})
    n = 2 * max(windows) + 90
    tokens = {"p": zt.random_tokens(tm.cfg, n, 12)}
    first = max(windows) + 1
    cuts = [c for c in [windows[0] - 1, 1, 1, first - windows[0] - 1, 2, 15, 1, 16] if c > 0]
    for page in (16, 64):
        steps = _portions(tokens["p"], cuts + [1] * (n - sum(cuts)))
        tm.check(tokens, harness.replay(tm.runner(-(-n // page) + 1, page=page), steps), f"{key} sharp x{sharp:g}")
    # the sharpening does what it is for: these mistakes move the logits
    right = tm.plain_logits(tokens["p"])

    def moved(change) -> float:
        cfg = json.loads(json.dumps(tm.cfg))
        for entry in cfg["layers"]:
            if entry["mixer"].get("mask"):
                change(entry["mixer"]["mask"])
        return zt.relative_error(plain.forward(cfg, tm.plain_weights, tokens["p"]), right)

    bar = 50 * zt.TOLERANCE["float32"]
    assert moved(lambda m: m.update(size=m["size"] - 1)) > bar and moved(lambda m: m.update(size=m["size"] + 1)) > bar
    assert moved(lambda m: m.update(keep_first=m["keep_first"] - 1)) > bar
    assert moved(lambda m: m.update(keep_first=m["keep_first"] + 1)) > bar
    bare = {k: torch.full_like(v, -1e4) if k.endswith("mix.sink") else v for k, v in tm.plain_weights.items()}
    assert zt.relative_error(plain.forward(tm.cfg, bare, tokens["p"]), right) > bar


@pytest.mark.parametrize("key", ["A", "B", "C"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_and_reused_pages_and_slots(key, dtype):
    """Up to three live requests of unequal lengths, portions beside single tokens, requests that pause, end and are
    followed by new ones in the same slots and pages (the pool is as small as the schedule allows)."""
    tm = _model(key, dtype)
    page = tm.page
    runner = tm.runner(3 * (-(-100 // page) + 1), slots=3)
    lengths = {"a": 100, "b": 37, "c": 64, "d": 90, "e": 3, "f": 45}
    tokens = {r: zt.random_tokens(tm.cfg, n, 10 + i) for i, (r, n) in enumerate(lengths.items())}
    fed = {r: 0 for r in lengths}

    def take(r, n):
        n = min(n, lengths[r] - fed[r])
        part = tokens[r][fed[r]: fed[r] + n]
        fed[r] += n
        return (r, part, list(range(n)))

    steps = []

    def step(*parts):
        entries = [take(r, n) for r, n in parts if fed[r] < lengths[r]]
        ends = [r for r, _, _ in entries if fed[r] == lengths[r]]
        if entries:
            steps.append((entries, ends))

    step(("a", 30), ("b", 2))
    step(("a", 1), ("b", 33), ("c", 17))
    step(("b", 1), ("c", 2))
    step(("a", 50), ("b", 1))            # b ends: its slot and pages go to d
    step(("a", 1), ("c", 40), ("d", 16))
    for _ in range(6):
        step(("a", 1), ("c", 1), ("d", 1))
    step(("a", 19), ("d", 2))            # a ends
    step(("c", 5), ("d", 60), ("e", 3))  # c, e end (e within one step)
    step(("d", 11), ("f", 44))
    step(("d", 1), ("f", 1))
    assert all(fed[r] == lengths[r] for r in lengths)
    got = harness.replay(runner, steps)
    tm.check(tokens, got, f"{key} mixed")
    stats = runner.cache.stats()
    assert stats["slots_used"] == 0 and all(g["used"] == 0 for g in stats["groups"])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_batch_equals_each_request_alone(dtype):
    tm = _model("C", dtype)
    tokens = {r: zt.random_tokens(tm.cfg, n, 20 + i) for i, (r, n) in enumerate({"a": 50, "b": 9, "c": 33}.items())}
    alone = {}
    for r, t in tokens.items():
        alone.update(harness.replay(tm.runner(8), [([(r, t[:-3], [len(t) - 4])], [])] +
                                    [([(r, [t[i]], [0])], []) for i in range(len(t) - 3, len(t))]))
    runner = tm.runner(16)
    steps = [([(r, t[:-3], [len(t) - 4]) for r, t in tokens.items()], [])]
    steps += [([(r, [t[len(t) - 3 + i]], [0]) for r, t in tokens.items()], []) for i in range(3)]
    together = harness.replay(runner, steps)
    errors = []
    for r in tokens:
        for position, row in alone[r].items():
            if dtype == "float32":
                assert torch.equal(row, together[r][position])
            else:
                errors.append(zt.relative_error(together[r][position], row))
    if errors:
        errors.sort()
        assert errors[-1] < 0.25 and errors[len(errors) // 2] < 2e-2, errors[-5:]


@pytest.mark.parametrize("key", ["A", "B"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(key, dtype):
    """400 tokens one by one: pages between the kept tokens and the window are given back and used again, while the
    first tokens stay in reach and the memories carry on."""
    tm = _model(key, dtype)
    runner = tm.runner(26)
    tokens = {"p": zt.random_tokens(tm.cfg, 400, 30)}
    steps = [([("p", tokens["p"][:4], [3])], [])]
    steps += [([("p", [tokens["p"][i]], [0] if i % 9 == 0 or i > 390 else [])], []) for i in range(4, 400)]
    tm.check(tokens, harness.replay(runner, steps), f"{key} long decoding")


def test_a_far_token_is_still_seen():
    """Two prompts that differ in their first token only: 300 tokens on, past every window, the logits still differ (kept
    tokens, latents and memories hold it), and the engine reproduces the difference, in a prompt and in a decoded token."""
    tm = _model("A", "float32", sharp=3.0)
    base = zt.random_tokens(tm.cfg, 301, 40)
    other = [(base[0] + 1) % tm.cfg["vocab"]] + base[1:]
    tokens = {"x": base, "y": other}
    got = harness.replay(tm.runner(48), [([("x", base[:300], [299]), ("y", other[:300], [299])], []),
                                         ([("x", base[300:], [0]), ("y", other[300:], [0])], ["x", "y"])])
    tm.check(tokens, got, "A far token")
    for position in (299, 300):
        want = tm.plain_logits(base)[position] - tm.plain_logits(other)[position]
        assert want.abs().max() > 1e-3
        assert zt.relative_error(got["x"][position] - got["y"][position], want) < 0.05


def test_sizes_come_from_the_configuration():
    """Values that a given model may leave equal to one another or at 1: one head, one kv head for many query heads, a
    window of 1 (a token sees itself and the kept ones), every token kept, a latent of one column, key and value sizes of
    1, one expert of one, a scale of 1, a pair table of one bucket, no feed-forward anywhere else."""
    cfg = zt.config(50, 32, 1e-3, (1.0, 1.0), (1, 1, 1), [
        zt.windowed(1, 1, 8, 4, None, size=1, keep_first=1, scale=1.0),
        zt.windowed(5, 1, 8, 12, zt.routed(8, 1, 1), size=2, keep_first=500),
        zt.latent(1, 3, 5, 1, 1, None, scale=1.0),
        zt.memory(1, 1, 1, zt.dense(8), cap=1.0),
        zt.latent(7, 1, 2, 3, 1, None, kv_from=2, scale=1.0),
        zt.memory(6, 16, 4, None, cap=30.0),
        zt.windowed(4, 1, 24, 12, zt.dense(8), size=3)], positions=40)
    for dtype in ("float32", "bfloat16"):
        tm = zt.TinyZemarax("-", dtype, cfg=cfg)
        tokens = {"p": zt.random_tokens(cfg, 40, 50)}
        steps = [([("p", tokens["p"][:20], list(range(20)))], [])]
        steps += [([("p", [t], [0])], []) for t in tokens["p"][20:]]
        tm.check(tokens, harness.replay(tm.runner(8), steps), "sizes of one")


def test_odd_sizes_and_a_larger_model():
    """A width that is no multiple of four with sizes that are no multiples of eight (every kernel's plain form), a model of
    wider rows (windows over several pages, kept tokens over page borders, latents of 96 and 112, memories of 128 x 256 and
    64 x 192), and rows and latents wider than the tensor-core kernels take."""
    small = zt.config(101, 70, 1e-5, (2.5, 1.3), (37, 5, 3), [
        zt.memory(3, 10, 6, zt.routed(30, 7, 3, 18), cap=3.0),
        zt.windowed(6, 3, 14, 6, zt.dense(50), size=13, keep_first=2),
        zt.latent(3, 22, 6, 9, 15, zt.routed(10, 9, 4)),
        zt.latent(5, 7, 11, 13, 15, None, kv_from=2)])
    large = zt.config(300, 200, 1e-6, (5.0, 2.5), (509, 97, 11), [
        zt.windowed(8, 2, 80, 48, zt.routed(48, 12, 4, 72), size=200, keep_first=33),
        zt.memory(2, 128, 256, zt.dense(352)),
        zt.latent(6, 48, 64, 72, 96, zt.dense(352)),
        zt.windowed(4, 2, 64, 128, zt.routed(64, 8, 2, 40), size=150, keep_first=70),
        zt.latent(10, 64, 32, 40, 96, None, kv_from=2),
        zt.latent(4, 64, 32, 40, 112, None),
        zt.memory(3, 64, 192, zt.dense(100), cap=7.0)])
    wide = zt.config(90, 48, 1e-5, (1.0, 1.0), (11, 2, 9), [
        zt.windowed(2, 1, 160, 40, zt.dense(64), size=30, keep_first=4, scale=0.1),
        zt.latent(20, 24, 20, 30, 144, None, scale=0.1),
        zt.memory(1, 300, 20, None)])
    for cfg, length in ((small, 120), (large, 450), (wide, 100)):
        for dtype in ("float32", "bfloat16"):
            tm = zt.TinyZemarax("-", dtype, cfg=cfg, seed=3)
            tokens = {"p": zt.random_tokens(cfg, length, 50), "q": zt.random_tokens(cfg, 77, 51)}
            p, q, cut = tokens["p"], tokens["q"], length - 40
            steps = [([("p", p[:cut], list(range(0, cut, 7)))], []),
                     ([("q", q[:70], [0, 69]), ("p", p[cut: cut + 1], [0])], [])]
            steps += [([("p", [p[i]], [0])] + ([("q", [q[70 + i - cut - 1]], [0])] if i - cut - 1 < 7 else []), [])
                      for i in range(cut + 1, length)]
            tm.check(tokens, harness.replay(tm.runner(64), steps), "odd sizes and a larger model")


def _random_config(seed: int):
    """Sizes, constants and layer order drawn at random."""
    gen = torch.Generator().manual_seed(3000 + seed)

    def pick(options):
        return options[int(torch.randint(0, len(options), (1,), generator=gen))]

    def feed_forward():
        choice = pick(["none", "dense", "dense", "moe", "moe"])
        if choice == "none":
            return None
        if choice == "dense":
            return zt.dense(pick([40, 72, 130]))
        experts = pick([1, 2, 4, 6, 9])
        return zt.routed(pick([8, 24, 40]), experts, pick(list(range(1, experts + 1))), pick([None, 16, 48]))

    width = pick([36, 52, 64, 100, 136])
    layers, sources = [], {}
    for i in range(pick([3, 4, 5, 6])):
        kind = pick(["attention", "mlstm", "latent", "latent"])
        if kind == "attention":
            kv = pick([1, 2, 3])
            window = pick([None, 1, 2, 5, 16, 17, 31, 33, 50])
            layers.append(zt.windowed(kv * pick([1, 2, 3, 4]), kv, pick([8, 12, 16, 32, 64]), pick([4, 8, 24, 64]), feed_forward(),
                                      size=window, keep_first=pick([0, 1, 4, 16, 17, 40]), scale=pick([0.1, 0.3, 1.0])))
        elif kind == "mlstm":
            layers.append(zt.memory(pick([1, 2, 3]), pick([4, 8, 16, 20, 32, 64]), pick([4, 6, 8, 16, 40, 72]), feed_forward(),
                                    cap=pick([1.5, 5.0, 15.0])))
        else:
            source = pick([None, *sources]) if sources else None
            rank = sources[source] if source is not None else pick([8, 20, 32, 48, 64])
            if source is None:
                sources[i] = rank
            layers.append(zt.latent(pick([1, 2, 3, 5]), pick([4, 8, 16, 24]), pick([4, 8, 24]), pick([6, 16, 40]), rank,
                                    feed_forward(), kv_from=source, scale=pick([0.1, 0.5, 1.0])))
    return zt.config(pick([64, 101, 257]), width, pick([1e-6, 1e-5, 1e-3]), (pick([1.0, 3.0, 12.0]), pick([1.0, 0.5, 3.0])),
                     (pick([1, 17, 2039]), pick([1, 211, 100003]), pick([1, 13, 65537])), layers, positions=pick([70, 128, 1000]))


@pytest.mark.parametrize("seed", list(range(12)))
def test_configurations_drawn_at_random(seed):
    """Each drawn model under a mixed schedule (portions, single tokens, a request that ends and one that takes its
    slot), float32 and bfloat16 against the plain implementation."""
    cfg = _random_config(seed)
    page = [16, 32, 64][seed % 3]
    for dtype in ("float32", "bfloat16"):
        tm = zt.TinyZemarax("-", dtype, seed=seed, cfg=cfg)
        tokens = {r: zt.random_tokens(cfg, n, 100 + seed + i) for i, (r, n) in enumerate({"a": 70, "b": 23, "c": 41}.items())}
        a, b, c = tokens["a"], tokens["b"], tokens["c"]
        steps = [([("a", a[:35], list(range(35))), ("b", b[:2], [0, 1])], []),
                 ([("a", a[35:36], [0]), ("b", b[2:23], list(range(21)))], ["b"]),
                 ([("a", a[36:37], [0]), ("c", c[:3], [0, 1, 2])], []),
                 ([("c", c[3:40], list(range(37))), ("a", a[37:38], [0])], [])]
        steps += [([("a", [a[i]], [0])] + ([("c", [c[40]], [0])] if i == 38 else []), ["c"] if i == 38 else [])
                  for i in range(38, 70)]
        runner = tm.runner(-(-70 // page) + -(-41 // page) + 2, slots=2, page=page)
        tm.check(tokens, harness.replay(runner, steps), f"random configuration {seed}")


def test_missing_and_misshapen_tensors_are_named():
    from pulsarlm_b200.engine.loading import load_model
    from pulsarlm_b200.weights.loader import WeightsError

    cfg, _ = zt.CONFIGS["A"]
    weights = zt.random_weights(cfg, 1)
    del weights["l1.mix.f.b"]
    weights["l0.mix.sink"] = weights["l0.mix.sink"][:-1].contiguous()
    tm = zt.TinyZemarax("A", "float32", weights=weights)
    with pytest.raises((WeightsError, ValueError)) as error:
        load_model(tm.folder, "float32", DEV)
    assert "l1.mix.f.b" in str(error.value) or "l0.mix.sink" in str(error.value)


# --------------------------------------------------------------------------- the engine

def _plain_greedy(tm, prompt, n_new):
    tokens = list(prompt)
    for _ in range(n_new):
        tokens.append(int(tm.plain_logits(tokens)[-1].argmax()))
    return tokens[len(prompt):]


@pytest.mark.parametrize("cuda_graphs", [False, True])
def test_greedy_generation_through_the_engine(cuda_graphs):
    """Requests of unequal lengths through Engine.submit / step: admission, prompt portions of 16 tokens beside decoding
    requests, more requests than slots (so slots and pages are used again), eager and captured decode steps; float32
    tokens equal the plain implementation's."""
    from pulsarlm_b200.engine.engine import Engine

    tm = _model("A", "float32")
    engine = Engine(tm.folder, dtype="float32", device=DEV, page_size=16, n_pages=40, max_requests=3,
                    prefill_tokens_per_step=16, cuda_graphs=cuda_graphs)
    prompts = [zt.random_tokens(tm.cfg, n, 60 + i) for i, n in enumerate([40, 3, 21, 1, 30])]
    requests = [engine.submit(p, max_tokens=25, ignore_eos=True) for p in prompts]
    for _ in range(600):
        if not engine.has_work():
            break
        engine.step()
    assert not engine.has_work()
    for prompt, request in zip(prompts, requests):
        assert list(request.output) == _plain_greedy(tm, prompt, 25)
    if cuda_graphs:
        assert engine.runner.graph_steps > 0


def test_engine_preempts_and_recomputes_the_states():
    """So few pages that running requests are preempted (pages and state slots given back, the request recomputed from
    its start later): the tokens are still the plain implementation's."""
    from pulsarlm_b200.engine.engine import Engine

    cfg, _ = zt.CONFIGS["B"]
    tm = zt.TinyZemarax("-", "float32", seed=4, cfg=cfg)
    engine = Engine(tm.folder, dtype="float32", device=DEV, page_size=16, n_pages=7, max_requests=4,
                    prefill_tokens_per_step=16)
    prompts = [zt.random_tokens(cfg, n, 95 + i) for i, n in enumerate([30, 25, 20])]
    requests = [engine.submit(p, max_tokens=20, ignore_eos=True) for p in prompts]
    for _ in range(600):
        if not engine.has_work():
            break
        engine.step()
    assert not engine.has_work() and engine.scheduler.preemptions > 0
    for prompt, request in zip(prompts, requests):
        assert request.finish_reason == "length"
        assert list(request.output) == _plain_greedy(tm, prompt, 20)


def test_engine_stops_at_the_last_position():
    """A model with a table of 40 positions: a request ends when its sequence is as long as the table (the last token
    drawn needs no position), a longer prompt is refused, and so is a step past the end."""
    from pulsarlm_b200.engine.engine import Engine
    from pulsarlm_b200.engine.runner import StepEntry

    cfg = zt.config(60, 32, 1e-5, (2.0, 1.0), (7, 3, 5), [zt.windowed(2, 1, 16, 16, zt.dense(24), size=8, keep_first=2),
                                                         zt.memory(2, 16, 16, None)], positions=40)
    for dtype in ("float32", "bfloat16"):
        tm = zt.TinyZemarax("-", dtype, cfg=cfg)
        engine = Engine(tm.folder, dtype=dtype, device=DEV, page_size=16, n_pages=20, max_requests=2, prefill_tokens_per_step=16)
        prompt = zt.random_tokens(cfg, 30, 3)
        requests = [engine.submit(prompt, ignore_eos=True), engine.submit(prompt[:5], max_tokens=500, ignore_eos=True)]
        for _ in range(200):
            if not engine.has_work():
                break
            engine.step()
        assert not engine.has_work()
        assert [len(r.output) for r in requests] == [11, 36] and all(r.finish_reason == "length" for r in requests)
        if dtype == "float32":
            assert list(requests[0].output) == _plain_greedy(tm, prompt, 11)
        with pytest.raises(ValueError):
            engine.submit(zt.random_tokens(cfg, 41, 4))
        runner = tm.runner(8)
        runner.step([StepEntry("p", zt.random_tokens(cfg, 40, 5), [39])])
        with pytest.raises(ValueError):
            runner.step([StepEntry("p", [1], [0])])


def test_captured_bfloat16_steps_equal_eager_ones():
    """Decode steps of several requests replayed from a capture (padding rows beside them) draw the tokens the eager
    steps draw, and their logits stay close to the plain implementation's."""
    from pulsarlm_b200.engine.engine import Engine

    tm = _model("C", "bfloat16")
    prompts = [zt.random_tokens(tm.cfg, n, 70 + i) for i, n in enumerate([50, 7, 33])]
    outputs = []
    for cuda_graphs in (False, True):
        engine = Engine(tm.folder, dtype="bfloat16", device=DEV, page_size=16, n_pages=40, max_requests=4,
                        prefill_tokens_per_step=128, record_logits=not cuda_graphs, cuda_graphs=cuda_graphs)
        requests = [engine.submit(p, max_tokens=20, ignore_eos=True) for p in prompts]
        while engine.has_work():
            engine.step()
        outputs.append([list(r.output) for r in requests])
        if not cuda_graphs:
            errors = []
            for prompt, request in zip(prompts, requests):
                ref = tm.plain_logits((list(prompt) + list(request.output))[:-1])
                errors += [zt.relative_error(row, ref[len(prompt) - 1 + i]) for i, row in enumerate(request.logits)]
            errors.sort()
            assert errors[len(errors) // 2] < 6e-2 and errors[-3] < 0.25
        else:
            assert engine.runner.graph_steps > 0
    agree = sum(a == b for x, y in zip(*outputs) for a, b in zip(x, y))
    assert agree >= 0.9 * sum(len(x) for x in outputs[0])   # (padding may change a batch's split counts: a rounding)


def _write(path, text) -> str:
    with open(path, "w") as f:
        json.dump(text, f)
    return str(path)


def test_command_line_random_model_generate_and_replay(tmp_path, capsys):
    """`models list`, `models random`, `generate` and the trace replay of the command line for this architecture: greedy
    tokens equal the plain implementation's on the written weights, and the replayed logits too."""
    import io

    import numpy as np
    from safetensors.torch import load_file

    from pulsarlm_b200 import cli
    from pulsarlm_b200.engine import trace

    assert cli.main(["models", "list"]) == 0
    assert "Zemarax" in capsys.readouterr().out.split()
    cfg, _ = zt.CONFIGS["C"]
    folder = str(tmp_path / "model")
    assert cli.main(["models", "random", folder, "--config", _write(tmp_path / "c.json", cfg), "--seed", "3",
                     "--dtype", "float32", "--std", "0.3"]) == 0
    capsys.readouterr()
    weights = {k: v.double() for k, v in load_file(folder + "/model.safetensors").items()}
    assert set(weights) == set(zt.tensor_shapes(cfg))
    prompt = zt.random_tokens(cfg, 19, 90)
    assert cli.main(["generate", folder, "--dtype", "float32", "--prompt_ids", ",".join(map(str, prompt)),
                     "--max_tokens", "8", "--ignore_eos"]) == 0
    record = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    tokens = list(prompt)
    for _ in range(8):
        tokens.append(int(plain.forward(cfg, weights, tokens)[-1].argmax()))
    assert record["output_ids"] == tokens[len(prompt):]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": tokens[:11], "want": [3, 10]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": tokens[:2], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": tokens[11:12], "want": [0]},
                                     {"id": "b", "tokens": tokens[2:9], "want": [6]}], "end": ["a", "b"]}]
    out = io.StringIO()
    assert trace.run(["--model", folder, "--dtype", "float32", "--out", str(tmp_path / "out"), "--max-tokens", "128"],
                     stdin=io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"), stdout=out) == 0
    assert out.getvalue().split() == ["done", "0", "done", "1", "done", "2"]
    ref = plain.forward(cfg, weights, tokens[:12])
    got0 = torch.from_numpy(np.fromfile(str(tmp_path / "out" / "0.f32"), dtype="<f4").reshape(2, -1))
    got2 = torch.from_numpy(np.fromfile(str(tmp_path / "out" / "2.f32"), dtype="<f4").reshape(2, -1))
    assert zt.relative_error(got0, ref[[3, 10]]) < 2e-4 and zt.relative_error(got2, ref[[11, 8]]) < 2e-4
    assert not (tmp_path / "out" / "1.f32").exists()
