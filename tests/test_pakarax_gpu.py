"""The Pakarax decoder in the engine against the plain implementation (plain_pakarax.py): each mechanism's kernel
alone, then whole models under every kind of schedule."""

from __future__ import annotations

import json

import pytest
import torch

import harness
import pakarax_tiny as pt
import plain_pakarax as plain

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


# --------------------------------------------------------------------------- mechanisms alone

@pytest.mark.parametrize("heads,kv,dim,vdim", [(4, 2, 16, 24), (3, 3, 10, 6), (2, 1, 40, 40), (8, 2, 64, 32), (1, 1, 5, 12)])
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_filtered_queries_keys_and_values_on_the_way_to_the_cache(heads, kv, dim, vdim, taps, dtype):
    """Two sequences in portions that need the state slot, then single tokens that move it on in the same launch; rows of
    a common size with zeros past their own columns; a temperature on the queries; pages in a scrambled order; columns
    of a wider product; slots that held something else before."""
    from pulsarlm_b200.parts.filtered_attention import stacked_rows

    ops = _ops()
    gen = torch.Generator().manual_seed(heads * 100 + dim + taps)
    page, coef, every = 8, 0.7, 5
    row = -(-max(dim, vdim) // 16) * 16
    sizes = (heads * dim, kv * dim, kv * vdim)
    starts, width = [], 0
    for n in sizes:
        starts.append(width)
        width += -(-n // 8) * 8
    lengths = [330, 29]
    slots = [2, 0]
    u = [(torch.randn(n, width + 8, generator=gen)).to(dtype) for n in lengths]
    bias = [torch.randn(n, generator=gen) for n in sizes]
    conv = [torch.randn(n, taps, generator=gen) for n in sizes]
    want = []
    for e in range(2):
        parts = [plain.filtered(u[e][:, at: at + n].double() + b.double(), c.double())
                 for at, n, b, c in zip(starts, sizes, bias, conv)]
        parts[0] = parts[0] * plain.query_temperature(torch.arange(lengths[e]), coef, every)[:, None]
        want.append([parts[0].view(-1, heads, dim), parts[1].view(-1, kv, dim), parts[2].view(-1, kv, vdim)])
    n_pages, table = _paged(lengths, page, gen)
    k_pool = torch.full((n_pages, kv, page, row), 7.0, dtype=dtype, device=DEV)
    v_pool = torch.full_like(k_pool, 7.0)
    state = torch.full((4, taps - 1, width), 3.0, dtype=dtype, device=DEV)
    stacked_bias = stacked_rows(bias)[0].to(DEV)
    stacked_conv = stacked_rows(conv)[0].t().contiguous().to(DEV)
    fed = [0, 0]
    bar = _bar(dtype)
    for step in ([(0, 4), (1, 2)], [(0, 2), (1, 3)], [(1, 1), (0, 1)], [(0, 1)], [(0, 302), (1, 20)], [(0, 1), (1, 1)],
                 [(1, 2), (0, 11)], [(0, 1)]):
        rows, pos, entry = [], [], []
        for e, (r, n) in enumerate(step):
            n = min(n, lengths[r] - fed[r])
            rows.append(u[r][fed[r]: fed[r] + n])
            pos += list(range(fed[r], fed[r] + n))
            entry += [e] * n
            fed[r] += n
        proj = torch.cat(rows).to(DEV)
        tokens = proj.shape[0]
        single = tokens == len(step)
        q = torch.full((tokens, heads, row), 7.0, dtype=dtype, device=DEV)
        entry_t, slots_t = _i32(entry), _i32([slots[r] for r, _ in step])
        ops.conv_qkv_write(proj[:, :width], width + 8, stacked_bias, stacked_conv, state, slots_t, single, coef, every,
                           _i32(pos), entry_t, table[[r for r, _ in step]].to(DEV), q, k_pool, v_pool, page, kv, dim, vdim,
                           starts[1], starts[2])
        if taps > 1 and not single:
            counts = [entry.count(e) for e in range(len(step))]
            firsts = [sum(counts[:e]) for e in range(len(step))]
            ops.filter_state(proj[:, :width], width + 8, _i32(firsts), _i32(counts), slots_t, state)
        want_q = torch.stack([want[step[e][0]][0][p] for e, p in zip(entry, pos)])
        assert plain.relative_error_of(q[:, :, :dim].cpu(), want_q) < bar, step
        assert row == dim or float(q[:, :, dim:].abs().max()) == 0.0
    for e in range(2):
        assert fed[e] <= lengths[e]
        for p in range(fed[e]):
            at = (int(table[e, p // page]), slice(None), p % page)
            got_k, got_v = k_pool[at].cpu(), v_pool[at].cpu()
            assert plain.relative_error_of(got_k[:, :dim], want[e][1][p]) < bar
            assert plain.relative_error_of(got_v[:, :vdim], want[e][2][p]) < bar
            assert float(got_k[:, dim:].abs().sum()) == 0.0 == float(got_v[:, vdim:].abs().sum())


def _attention_case(gen, lengths, heads, kv, dim, page, dtype, spike_at, queries):
    """Paged keys and values of some requests and queries for chosen (request, position) pairs; a key at distance
    `spike_at` of every query lined up with the query of the flattest head so that it dominates despite the distance."""
    n_pages, table = _paged(lengths, page, gen)
    keys = [torch.randn(n, kv, dim, generator=gen).to(dtype) for n in lengths]
    values = [torch.randn(n, kv, dim, generator=gen).to(dtype) for n in lengths]
    q_full = [torch.randn(n, heads, dim, generator=gen).to(dtype) for n in lengths]
    if spike_at is not None:
        for e, p in queries:
            if p - spike_at >= 0:
                direction = q_full[e][p, heads - 1].float() / q_full[e][p, heads - 1].float().norm()
                keys[e][p - spike_at, kv - 1] = (40.0 * direction).to(dtype)
    both = torch.zeros(n_pages, 2, kv, page, dim, dtype=dtype, device=DEV)
    for e, n in enumerate(lengths):
        for j in range(n):
            both[table[e, j // page], 0, :, j % page] = keys[e][j].to(DEV)
            both[table[e, j // page], 1, :, j % page] = values[e][j].to(DEV)
    return table, keys, values, q_full, both


@pytest.mark.parametrize("heads,kv,dim", [(6, 2, 16), (2, 2, 20), (64, 64, 8)])
@pytest.mark.parametrize("spike", [None, 1, 16, 150])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_slopes_and_sinks_on_the_cuda_core_kernel(heads, kv, dim, spike, dtype):
    ops = _ops()
    page, scale = 8, 0.3
    lengths = [170, 33, 8, 129]
    gen = torch.Generator().manual_seed(11)
    queries = [(e, p) for e, n in enumerate(lengths) for p in sorted({0, 1, 2, 7, 8, n // 2, n - 2, n - 1}) if 0 <= p < n]
    table, keys, values, q_full, both = _attention_case(gen, lengths, heads, kv, dim, page, dtype, spike, queries)
    sinks = 2.0 * torch.randn(heads, generator=gen)
    q = torch.stack([q_full[e][p] for e, p in queries]).to(DEV)
    slopes = torch.tensor(plain.slopes(heads), dtype=torch.float32, device=DEV)
    for sink in (sinks, None):
        full = [plain.sloped_attention(q_full[e].double(), keys[e].double(), values[e].double(), scale,
                                       sink.double() if sink is not None else None) for e in range(len(lengths))]
        want = torch.stack([full[e][p] for e, p in queries])
        out = torch.empty_like(q)
        ops.attention_simt(q, both[:, 0], both[:, 1], table.to(DEV), _i32([p for _, p in queries]),
                           _i32([e for e, _ in queries]), out, page, None, scale,
                           sinks=sink.to(DEV) if sink is not None else None, distance_slopes=slopes)
        assert plain.relative_error_of(out.cpu(), want) < _bar(dtype)


@pytest.mark.parametrize("heads,kv,dim", [(6, 2, 32), (4, 1, 96), (3, 3, 64), (4, 2, 64), (8, 1, 128), (5, 1, 128), (16, 1, 48)])
@pytest.mark.parametrize("spike", [None, 1, 64, 190])
def test_slopes_and_sinks_on_the_tensor_core_kernels(heads, kv, dim, spike):
    """The bfloat16 kernels for single tokens (any number of key shares) and prompt portions (mma.sync; tcgen05 with
    heads in pairs and, for odd groups, with two halves of a tile; keys split among CTAs)."""
    ops = _ops()
    page, scale, dtype = 16, 0.25, torch.bfloat16
    lengths = [500, 33, 16, 129]
    slopes = torch.tensor(plain.slopes(heads), dtype=torch.float32, device=DEV)

    def case(queries, seed):
        gen = torch.Generator().manual_seed(seed)
        table, keys, values, q_full, both = _attention_case(gen, lengths, heads, kv, dim, page, dtype, spike, queries)
        sinks = 2.0 * torch.randn(heads, generator=gen)
        full = [plain.sloped_attention(q_full[e].double(), keys[e].double(), values[e].double(), scale, sinks.double())
                for e in range(len(lengths))]
        q = torch.stack([q_full[e][p] for e, p in queries]).to(DEV)
        return q, both, table.to(DEV), sinks.to(DEV), torch.stack([full[e][p] for e, p in queries])

    queries = [(e, n - 1) for e, n in enumerate(lengths)] + [(0, 0), (0, 1), (3, 64)]
    q, both, table, sinks, want = case(queries, 21)
    pos, entry = _i32([p for _, p in queries]), _i32([e for e, _ in queries])
    for splits in (1, 2, 5, 20):
        for split_weights in (False, True):
            scratch = torch.empty(ops.attention_decode_scratch_floats(len(queries), heads, dim, splits),
                                  dtype=torch.float32, device=DEV) if splits > 1 else None
            out = torch.empty_like(q)
            ops.attention_decode(q, both[:, 0], both[:, 1], table, pos, entry, out, page, None, scale, splits, scratch,
                                 extras=ops.attention_extras(q, sinks, None, split_weights, 0.0, None, slopes))
            assert plain.relative_error_of(out.cpu(), want) < 1e-2, ("single tokens", splits)
    spans = [(0, 120, 500), (3, 0, 129), (1, 31, 33), (2, 0, 16)]
    queries = [(e, p) for e, lo, hi in spans for p in range(lo, hi)]
    q, both, table, sinks, want = case(queries, 22)

    def tiles_of(rows):
        tiles, at = [], 0
        for e, lo, hi in spans:
            for r in range(0, hi - lo, rows):
                tiles.append((at + r, min(rows, hi - lo - r), lo + r, e))
            at += hi - lo
        return _i32(tiles)

    out = torch.empty_like(q)
    ops.attention_prefill(q, both[:, 0], both[:, 1], table, tiles_of(ops.attention_prefill_tile_rows()), out, page, None,
                          scale, extras=ops.attention_extras(q, sinks, None, False, 0.0, None, slopes))
    assert plain.relative_error_of(out.cpu(), want) < 1e-2, "prompt rows"
    if not ops.attention_prefill_tcgen05_supports(q, both[:, 0], page):
        return
    for rows in {ops.attention_prefill_tile_rows(), ops.attention_prefill_tcgen05_tile_rows(heads // kv)}:
        for splits in (1, 2, 3):
            scratch = torch.empty(ops.attention_prefill_scratch_floats(q.shape[0], heads, dim, splits), dtype=torch.float32,
                                  device=DEV) if splits > 1 else None
            out = torch.empty_like(q)
            ops.attention_prefill_tcgen05(q, both[:, 0], both[:, 1], table, tiles_of(rows), out, page, None, scale, None,
                                          splits, scratch, distance_slopes=slopes, sinks=sinks)
            assert plain.relative_error_of(out.cpu(), want) < 1e-2, ("prompt rows on tcgen05", rows, splits)


def _recurrence_part(width, blocks, taps, hidden, dtype, gen, lam=None, slots=3):
    from pulsarlm_b200.parts.linear_recurrence import LinearRecurrence
    from pulsarlm_b200.parts.registry import BuildContext
    from pulsarlm_b200.parts.spec import PartSpec

    block = width // blocks
    w = {"y": torch.randn(width, hidden, generator=gen) / hidden ** 0.5, "y.b": 0.3 * torch.randn(width, generator=gen),
         "x": torch.randn(width, hidden, generator=gen) / hidden ** 0.5, "x.b": 0.3 * torch.randn(width, generator=gen),
         "conv": torch.randn(width, taps, generator=gen) / taps ** 0.5, "conv.b": 0.3 * torch.randn(width, generator=gen),
         "ra": 2.0 * torch.randn(blocks, block, block, generator=gen) / block ** 0.5,
         "ra.b": 0.3 * torch.randn(blocks, block, generator=gen),
         "ri": 2.0 * torch.randn(blocks, block, block, generator=gen) / block ** 0.5,
         "ri.b": 0.3 * torch.randn(blocks, block, generator=gen),
         "lam": lam if lam is not None else -9.0 * torch.rand(width, generator=gen),
         "o": torch.randn(hidden, width, generator=gen) / width ** 0.5}
    w = {k: v.to(dtype) for k, v in w.items()}
    spec = PartSpec("linear_recurrence", {"hidden_size": hidden, "width": width, "blocks": blocks, "taps": taps},
                    {**{n: n for n in ("y", "x", "conv", "ra", "ri", "lam", "o")},
                     **{n + "_bias": n + ".b" for n in ("y", "x", "conv", "ra", "ri")}})
    part = LinearRecurrence(spec, BuildContext(dtype, torch.device(DEV)))
    part.load({k: v.to(DEV) for k, v in w.items()})

    class Binding:
        pass

    mine, ring = Binding(), Binding()
    mine.states = torch.zeros(slots, width, dtype=torch.float32, device=DEV)
    ring.states = torch.zeros(slots, taps, width, dtype=dtype, device=DEV)
    part.bind_cache(mine)
    part.ring.bind_cache(ring)
    return part, {k: v.double() for k, v in w.items()}


def _recurrence_step(part, entries, seqs, fed, slot_of):
    """One step of (sequence, tokens) entries, single tokens first as the step function orders them; returns
    {(sequence, position): row}."""
    from pulsarlm_b200.parts.delta_rule import SEQUENCE_ROWS_KEY

    class Batch:
        pass

    batch = Batch()
    rows, pos, entry, first, count = [], [], [], [], []
    for e, (r, n) in enumerate(entries):
        first.append(len(pos))
        count.append(n)
        rows.append(seqs[r][fed[r]: fed[r] + n])
        pos += list(range(fed[r], fed[r] + n))
        entry += [e] * n
    batch.pos, batch.entry, batch.slots = _i32(pos), _i32(entry), _i32([slot_of[r] for r, _ in entries])
    batch.n_decode = sum(1 for n in count if n == 1)
    batch.host_query_lens = count
    batch.plans = {SEQUENCE_ROWS_KEY: {"first": _i32(first), "count": _i32(count)}}
    out = part.forward(torch.cat(rows).to(DEV), batch).float().cpu()
    got = {}
    for row, e, p in zip(out, entry, pos):
        got[(entries[e][0], p)] = row
    for r, n in entries:
        fed[r] += n
    return got


@pytest.mark.parametrize("width,blocks,taps", [(64, 2, 3), (60, 5, 4), (33, 3, 2), (200, 1, 1), (160, 10, 6), (130, 2, 4)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_gated_recurrence_in_portions_and_token_by_token(width, blocks, taps, dtype):
    """Portions shorter and longer than what a CTA walks at once and than a cluster does, beside single tokens, single
    tokens alone, a slot that a second sequence takes over after the first (zeroed, as the cache manager does)."""
    _ops()
    gen = torch.Generator().manual_seed(width + taps)
    hidden = 40
    part, w = _recurrence_part(width, blocks, taps, hidden, dtype, gen)
    lengths = {"a": 1400, "b": 139, "c": 61}
    seqs = {r: torch.randn(n, hidden, generator=gen).to(dtype) for r, n in lengths.items()}
    slot_of = {"a": 2, "b": 0, "c": 0}

    def rnd(t):
        return t.to(dtype).double() if dtype == torch.bfloat16 else t

    want = {r: plain.right_branch(s.double(), w, {"blocks": blocks}, rnd) for r, s in seqs.items()}
    fed = {r: 0 for r in seqs}
    got = {}
    for step in ([("b", 1), ("a", 129)], [("a", 2), ("b", 2)], [("a", 1), ("b", 1)], [("a", 1), ("b", 100)],
                 [("b", 1), ("a", 1100)], [("b", 1)], [("a", 3), ("b", 30)], [("b", 1), ("a", 1)], [("b", 1), ("a", 1)],
                 [("b", 1)], [("a", 161)]):
        got.update(_recurrence_step(part, step, seqs, fed, slot_of))
    assert fed["b"] == 139
    part.states[0].zero_()
    part.ring.binding.states[0].zero_()
    for n in [1, 1, 2, 1, 20, 1, 33, 1, 1]:
        got.update(_recurrence_step(part, [("c", n)], seqs, fed, slot_of))
    for r in seqs:
        mine = torch.stack([got[(r, p)] for p in range(fed[r])])
        error = (mine.double() - want[r][: fed[r]]).abs().amax(dim=1) / want[r].abs().max()
        assert float(error.max()) < (2e-5 if dtype == torch.float32 else 2e-2), (r, int(error.argmax()))


def test_recurrence_keeps_what_a_slow_decay_keeps():
    """Channels whose state hardly decays: what the first tokens brought is still there 3,000 tokens on, and a short
    memory's is not; 1 - a^2 keeps its digits where a is near 1."""
    _ops()
    gen = torch.Generator().manual_seed(5)
    width, hidden, n = 64, 16, 3000
    lam = torch.cat([torch.full((32,), -14.0), torch.full((32,), 3.0)])
    seqs = {"a": torch.randn(n, hidden, generator=gen)}
    seqs["b"] = torch.cat([-3.0 * seqs["a"][:5], seqs["a"][5:]])
    part, w = _recurrence_part(width, 2, 4, hidden, torch.float32, gen, lam=lam)
    want = {r: plain.right_branch(s.double(), w, {"blocks": 2}, lambda t: t) for r, s in seqs.items()}
    fed = {"a": 0, "b": 0}
    got = {}
    for step in ([("a", 1500), ("b", 700)], [("a", 1), ("b", 800)], [("b", 1), ("a", 1000)], [("a", n - 2501), ("b", n - 1501)]):
        got.update(_recurrence_step(part, step, seqs, fed, {"a": 1, "b": 2}))
    for r in seqs:
        mine = torch.stack([got[(r, p)] for p in range(n)])
        assert plain.relative_error_of(mine, want[r]) < 2e-5
    last = got[("a", n - 1)].double() - got[("b", n - 1)].double()
    wanted = want["a"][-1] - want["b"][-1]
    assert float(wanted.abs().max()) > 1e-3 * float(want["a"].abs().max())
    assert float((last - wanted).abs().max()) < 0.02 * float(wanted.abs().max())


@pytest.mark.parametrize("hidden", [30, 72, 192, 2048, 2600, 9000])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_two_normed_sides_enter_the_stream(hidden, dtype):
    """With and without the third output, the biases and the sides; the next norm, chosen rows only, or the stream
    beside what entered the first layer."""
    ops = _ops()
    gen = torch.Generator().manual_seed(hidden)
    tokens, eps = 11, 1e-5
    x = torch.randn(tokens, hidden, generator=gen)
    y1, y2, y3 = ((torch.randn(tokens, hidden, generator=gen) * s).to(dtype) for s in (3.0, 0.01, 1.0))
    b1, b2, w1, w2, w = (torch.randn(hidden, generator=gen) for _ in range(5))
    entered = torch.randn(tokens, hidden, generator=gen)
    for biases in (True, False):
        for third in (True, False):
            for sides in (True, False):
                add = y3.double() if third else torch.zeros(tokens, hidden, dtype=torch.float64)
                if sides:
                    u1 = y1.double() + (b1.double() if biases else 0.0)
                    u2 = y2.double() + (b2.double() if biases else 0.0)
                    add = add + plain.side_by_side(u1, u2, w1.double(), w2.double(), eps)
                want = x.double() + add
                given = tuple(t.to(DEV) if t is not None else None for t in
                              (y1, b1 if biases else None, w1, y2, b2 if biases else None, w2)) if sides else None
                mine = y3.to(DEV) if third else None
                stream, out = x.to(DEV), torch.empty(tokens, hidden, dtype=dtype, device=DEV)
                ops.side_norm(stream, given, 0.5, eps, mine, w.to(DEV), 1e-4, out)
                normed = plain.rms(want, 1e-4) * w.double()
                assert plain.relative_error_of(stream.cpu(), want) < 1e-6
                assert plain.relative_error_of(out.cpu(), normed) < _bar(dtype)
                rows = [7, 0, 7]
                kept, out = x.to(DEV), torch.empty(3, hidden, dtype=dtype, device=DEV)
                ops.side_norm(kept, given, 0.5, eps, mine, w.to(DEV), 1e-4, out, _i32(rows))
                assert plain.relative_error_of(out.cpu(), normed[rows]) < _bar(dtype) and torch.equal(kept.cpu(), x)
                both = torch.empty(tokens, 2 * hidden, dtype=dtype, device=DEV)
                ops.side_norm(x.to(DEV), given, 0.5, eps, mine, None, 0.0, both, entered=entered.to(DEV))
                assert plain.relative_error_of(both.cpu(), torch.cat([want, entered.double()], dim=1)) < _bar(dtype)
                stream = x.to(DEV)
                ops.side_norm(stream, given, 0.5, eps, mine, None, 0.0, None)
                assert plain.relative_error_of(stream.cpu(), want) < 1e-6


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_projection_that_joins_the_stream_with_the_embedding(dtype):
    from pulsarlm_b200.parts.registry import BuildContext, build_part
    from pulsarlm_b200.parts.spec import PartSpec

    _ops()
    gen = torch.Generator().manual_seed(2)
    hidden = 48
    weight = (torch.randn(hidden, 2 * hidden, generator=gen) / hidden ** 0.5).to(dtype)
    part = build_part("join", PartSpec("concat_linear", {"hidden_size": hidden}, {"weight": "w"}),
                      BuildContext(dtype, torch.device(DEV)))
    part.load({"w": weight.to(DEV)})
    for tokens in (1, 5, 300):
        x, x0 = torch.randn(tokens, hidden, generator=gen), torch.randn(tokens, hidden, generator=gen)
        delta = torch.randn(tokens, hidden, generator=gen).to(dtype)
        got = part.forward(x.to(DEV), delta.to(DEV), x0.to(DEV))
        assert got.dtype == torch.float32
        want = torch.cat([x.double() + delta.double(), x0.double()], dim=1) @ weight.double().T
        assert plain.relative_error_of(got.cpu(), want) < _bar(dtype)


@pytest.mark.parametrize("width", [6, 24, 130])
@pytest.mark.parametrize("limit", [0.5, 2.0, 100.0])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_clamped_unit_with_and_without_row_weights(width, limit, dtype):
    ops = _ops()
    gen = torch.Generator().manual_seed(width)
    tokens = 37
    both = (3.0 * torch.randn(tokens, 2 * width, generator=gen)).to(dtype)
    weights = torch.rand(tokens + 3, generator=gen)
    index = torch.randint(0, tokens + 3, (tokens,), generator=gen)
    for w, idx in ((None, None), (weights, index), (weights[:tokens].contiguous(), None)):
        factor = torch.ones(tokens) if w is None else w[idx] if idx is not None else w
        g, u = factor[:, None].double() * both[:, :width].double(), factor[:, None].double() * both[:, width:].double()
        out = torch.empty(tokens, width, dtype=dtype, device=DEV)
        ops.gated_act(both.to(DEV), out, "clamped", limit, w.to(DEV) if w is not None else None,
                      idx.int().to(DEV) if idx is not None else None)
        assert plain.relative_error_of(out.cpu(), plain.clamped_unit(g, u, limit)) < _bar(dtype)


@pytest.mark.parametrize("experts,top", [(8, 2), (5, 1), (3, 3), (64, 6)])
@pytest.mark.parametrize("tokens", [3, 300])
@pytest.mark.parametrize("shared", [False, True])
def test_router_with_plain_sigmoid_weights_and_a_shared_gate(experts, top, tokens, shared):
    ops = _ops()
    gen = torch.Generator().manual_seed(experts)
    hidden = 40
    h, router = torch.randn(tokens, hidden, generator=gen), torch.randn(experts, hidden, generator=gen) * 0.5
    gate_row = torch.randn(1, hidden, generator=gen) * 0.5
    ids, weights = plain.route(h.double(), router.double(), top)
    gate = torch.empty(tokens, dtype=torch.float32, device=DEV) if shared else None
    rows = torch.cat([router, gate_row]) if shared else router
    got_ids, got_w = ops.moe_route(h.to(DEV), rows.to(DEV), None, top, 1, 1, True, 1, False, gate)
    assert torch.equal(got_ids.cpu().long(), ids)
    assert plain.relative_error_of(got_w.cpu(), weights) < 1e-5
    if shared:
        assert plain.relative_error_of(gate.cpu(), torch.sigmoid(h.double() @ gate_row.double().T)[:, 0]) < 1e-5


@pytest.mark.parametrize("tokens", [1, 5, 130])
@pytest.mark.parametrize("top,shared", [(1, (40, 0.7)), (3, (24, 2.0)), (2, None)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_experts_weighed_on_their_input(tokens, top, shared, dtype):
    """The feed-forward part alone, few tokens (every pair streams its expert) and many (grouped products). Limits that
    bite: a weight on the output instead would show."""
    from pulsarlm_b200.parts.registry import BuildContext, build_part
    from pulsarlm_b200.parts.spec import PartSpec

    _ops()
    gen = torch.Generator().manual_seed(3)
    td = torch.float32 if dtype == "float32" else torch.bfloat16
    width, ff, experts = 48, 24, 8
    mlp = pt.routed(ff, experts, top, 0.5, shared)
    w = {"router": torch.randn(experts, width, generator=gen) * 0.5}
    sizes = {f"e{e}.": ff for e in range(experts)}
    if shared:
        sizes["shared."] = shared[0]
        w["shared.sg"] = torch.randn(1, width, generator=gen) / width ** 0.5
    for n, size in sizes.items():
        for leaf in ("gate", "up"):
            w[n + leaf] = 2.0 * torch.randn(size, width, generator=gen) / width ** 0.5
        w[n + "down"] = torch.randn(width, size, generator=gen) / size ** 0.5
    w = {k: v.to(td) for k, v in w.items()}
    h = torch.randn(tokens, width, generator=gen).to(td)
    want = plain.routed_ff(h.double(), {k: v.double() for k, v in w.items()}, mlp, lambda t: t)
    tensors = {"router": "router", "expert_gate": "e{e}.gate", "expert_up": "e{e}.up", "expert_down": "e{e}.down"}
    if shared:
        tensors.update(shared_gate="shared.gate", shared_up="shared.up", shared_down="shared.down",
                       shared_gate_row="shared.sg")
    spec = PartSpec("moe", {"hidden_size": width, "expert_size": ff, "n_experts": experts, "top": top,
                            "shared_size": shared[0] if shared else None, "scores": "sigmoid", "renormalise": False,
                            "expert": "clamped", "expert_limit": 0.5, "shared_limit": shared[1] if shared else None,
                            "weigh_input": True}, tensors)
    part = build_part("feed_forward", spec, BuildContext(td, torch.device(DEV)))
    part.load({k: v.to(DEV) for k, v in w.items()})
    assert plain.relative_error_of(part.forward(h.to(DEV), None).cpu(), want) < (1e-5 if dtype == "float32" else 2e-2)


@pytest.mark.parametrize("tokens", [1, 7, 40, 300])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_gated_feed_forward_with_the_clamped_unit(tokens, dtype):
    from pulsarlm_b200.parts.registry import BuildContext, build_part
    from pulsarlm_b200.parts.spec import PartSpec

    _ops()
    gen = torch.Generator().manual_seed(4)
    td = torch.float32 if dtype == "float32" else torch.bfloat16
    width, ff = 64, 136
    w = {"gate": 2.0 * torch.randn(ff, width, generator=gen) / 8.0, "up": 2.0 * torch.randn(ff, width, generator=gen) / 8.0,
         "down": torch.randn(width, ff, generator=gen) / ff ** 0.5}
    w = {k: v.to(td) for k, v in w.items()}
    h = torch.randn(tokens, width, generator=gen).to(td)
    part = build_part("feed_forward", PartSpec("gated_mlp", {"hidden_size": width, "intermediate_size": ff,
                                                             "activation": "clamped", "limit": 0.9}, {n: n for n in w}),
                      BuildContext(td, torch.device(DEV)))
    part.load({k: v.to(DEV) for k, v in w.items()})
    d = {k: v.double() for k, v in w.items()}
    want = plain.clamped_ff(h.double(), d["gate"], d["up"], d["down"], 0.9, lambda t: t)
    assert plain.relative_error_of(part.forward(h.to(DEV), None).cpu(), want) < (1e-5 if dtype == "float32" else 2e-2)


@pytest.mark.parametrize("tokens,ff", [(300, 200), (257, 136), (64, 512)])
def test_clamped_unit_in_the_epilogue_of_a_prompt_product(tokens, ff):
    """The pair kernel forms the unit from the rounded products, as the kernel alone does."""
    ops = _ops()
    gen = torch.Generator().manual_seed(ff)
    width, limit, bf = 96, 0.8, torch.bfloat16
    x = torch.randn(tokens, width, generator=gen).to(bf)
    gate_up = (2.0 * torch.randn(2 * ff, width, generator=gen) / width ** 0.5).to(bf)
    both = (x.double() @ gate_up.double().T).to(bf).double()
    want = plain.clamped_unit(both[:, :ff], both[:, ff:], limit)
    act = torch.empty(tokens, ff, dtype=bf, device=DEV)
    ops.gemm_bf16(x.to(DEV), gate_up.to(DEV), act, kernel="pair", gated=True, limit=limit)
    assert plain.relative_error_of(act.cpu(), want) < 1e-2


def test_scaled_and_capped_logits():
    ops = _ops()
    gen = torch.Generator().manual_seed(6)
    for shape in ((3, 101), (1, 7), (5, 4096)):
        x = 20.0 * torch.randn(shape, generator=gen)
        got = x.to(DEV)
        ops.capped_scale(got, 1.7, 12.0)
        assert plain.relative_error_of(got.cpu(), plain.capped(x.double() * 1.7, 12.0)) < 1e-6


# --------------------------------------------------------------------------- whole models

def _model(key, dtype, seed=1, sharp=1.0):
    return pt.TinyPakarax(key, dtype, seed, sharp=sharp)


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
    tokens = {"p": pt.random_tokens(tm.cfg, 175, 3), "q": pt.random_tokens(tm.cfg, 5, 4), "r": pt.random_tokens(tm.cfg, 1, 5)}
    got = harness.replay(runner, [([("p", tokens["p"], list(range(175)))], ["p"]),
                                  ([("q", tokens["q"], list(range(5)))], ["q"]),
                                  ([("r", tokens["r"], [0])], ["r"])])
    tm.check(tokens, got, f"{key} whole")


def test_residual_stream_after_every_layer():
    """float32: the stream after each layer run of a prompt fed in two portions, against the plain implementation's, so
    that a fault is placed at its layer."""
    from pulsarlm_b200.engine.runner import StepEntry
    from pulsarlm_b200.parts.basic import settle_pending

    for key in ("A", "B", "C"):
        tm = _model(key, "float32")
        tokens = pt.random_tokens(tm.cfg, 37, 9)
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
        runs = len(plain.layer_runs(tm.cfg))
        assert len(seen) == 2 * runs == 2 * len(want)
        for i in range(runs):
            got = torch.cat([seen[i], seen[runs + i]])
            assert plain.relative_error_of(got, want[i]) < 2e-5, (key, i)


@pytest.mark.parametrize("key", ["A", "B", "C"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prefill_then_token_by_token(key, dtype):
    """A prompt in one step, then 70 tokens one by one, over page borders."""
    tm = _model(key, dtype)
    runner = tm.runner(24)
    tokens = {"p": pt.random_tokens(tm.cfg, 110, 5)}
    steps = [([("p", tokens["p"][:40], [0, 1, 39])], [])]
    steps += [([("p", [tokens["p"][i]], [0])], []) for i in range(40, 110)]
    tm.check(tokens, harness.replay(runner, steps), f"{key} decode")


@pytest.mark.parametrize("key", ["A", "B", "C"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_token_by_token_from_the_start(key, dtype):
    """The first tokens of a sequence: convolutions that reach before its start, a state from zero."""
    tm = _model(key, dtype)
    runner = tm.runner(8)
    tokens = {"p": pt.random_tokens(tm.cfg, 30, 6)}
    steps = [([("p", [t], [0])], []) for t in tokens["p"]]
    tm.check(tokens, harness.replay(runner, steps), f"{key} from the start")


@pytest.mark.parametrize("key", ["A", "B", "C"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_of_many_sizes(key, dtype):
    tm = _model(key, dtype)
    runner = tm.runner(24)
    tokens = {"p": pt.random_tokens(tm.cfg, 300, 7)}
    cuts = [2, 2, 3, 1, 1, 7, 16, 2, 33, 1, 2, 17, 31, 2, 30, 129, 1, 2, 18]
    tm.check(tokens, harness.replay(runner, _portions(tokens["p"], cuts)), f"{key} portions")


@pytest.mark.parametrize("key", ["A", "B"])
def test_float32_bits_do_not_depend_on_the_cut(key):
    """In float32 every kernel adds in an order fixed by the token's own place: logits of a prompt fed whole and fed in
    portions are equal bit for bit."""
    tm = _model(key, "float32")
    tokens = pt.random_tokens(tm.cfg, 290, 8)
    whole = harness.replay(tm.runner(24), [([("p", tokens, list(range(290)))], [])])["p"]
    cut = harness.replay(tm.runner(24), _portions(tokens, [5, 1, 2, 40, 1, 1, 3, 37, 129, 71]))["p"]
    for position in range(290):
        assert torch.equal(whole[position], cut[position]), position


@pytest.mark.parametrize("key", ["A", "C"])
@pytest.mark.parametrize("sharp", [3.0, 6.0])
def test_sharp_attention_shows_every_key_in_reach(key, sharp):
    """float32, scores multiplied so that each softmax rests on a few keys: a far key lost with its page, a slope taken
    for another head's, a temperature that steps one token late or a sink left out would move these logits by orders
    more than the bar. Portions cut around page borders and temperature steps, then single tokens, with pages of 16
    and of 64."""
    tm = _model(key, "float32", seed=7, sharp=sharp)
    n = 130
    tokens = {"p": pt.random_tokens(tm.cfg, n, 12)}
    cuts = [15, 1, 1, 15, 2, 31, 1, 16]
    for page in (16, 64):
        steps = _portions(tokens["p"], cuts + [1] * (n - sum(cuts)))
        tm.check(tokens, harness.replay(tm.runner(-(-n // page) + 1, page=page), steps), f"{key} sharp x{sharp:g}")
    # the sharpening does what it is for: these mistakes move the logits
    right = tm.plain_logits(tokens["p"])
    late = json.loads(json.dumps(tm.cfg))
    for entry in late["layers"]:
        if entry["mixer"]["left"].get("q_temp"):
            entry["mixer"]["left"]["q_temp"]["every"] += 1
    assert pt.relative_error(plain.forward(late, tm.plain_weights, tokens["p"]), right) > 50 * pt.TOLERANCE["float32"]
    bare = {k: torch.full_like(v, -1e4) if k.endswith("left.sink") else v for k, v in tm.plain_weights.items()}
    assert pt.relative_error(plain.forward(tm.cfg, bare, tokens["p"]), right) > 50 * pt.TOLERANCE["float32"]


@pytest.mark.parametrize("key", ["A", "C"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_and_reused_pages_and_slots(key, dtype):
    """Up to three live requests of unequal lengths, portions beside single tokens, requests that pause, end and are
    followed by new ones in the same slots and pages (the pool is as small as the schedule allows)."""
    tm = _model(key, dtype)
    page = tm.page
    runner = tm.runner(3 * (-(-100 // page) + 1), slots=3)
    lengths = {"a": 100, "b": 37, "c": 64, "d": 90, "e": 3, "f": 45}
    tokens = {r: pt.random_tokens(tm.cfg, n, 10 + i) for i, (r, n) in enumerate(lengths.items())}
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
    tokens = {r: pt.random_tokens(tm.cfg, n, 20 + i) for i, (r, n) in enumerate({"a": 50, "b": 9, "c": 33}.items())}
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
                errors.append(pt.relative_error(together[r][position], row))
    if errors:
        errors.sort()
        assert errors[-1] < 0.25 and errors[len(errors) // 2] < 3e-2, errors[-5:]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(dtype):
    tm = _model("B", dtype)
    runner = tm.runner(16)
    tokens = {"p": pt.random_tokens(tm.cfg, 400, 30)}
    steps = [([("p", tokens["p"][:4], [3])], [])]
    steps += [([("p", [tokens["p"][i]], [0] if i % 9 == 0 or i > 390 else [])], []) for i in range(4, 400)]
    tm.check(tokens, harness.replay(runner, steps), "B long decoding")


def test_a_far_token_is_still_seen():
    """Two prompts that differ in their first token only: 300 tokens on the logits still differ (a flat head and a slow
    decay both reach that far), and the engine reproduces the difference, in a prompt and in a decoded token."""
    tm = _model("A", "float32", sharp=3.0)
    base = pt.random_tokens(tm.cfg, 301, 40)
    other = [(base[0] + 1) % tm.cfg["vocab"]] + base[1:]
    tokens = {"x": base, "y": other}
    got = harness.replay(tm.runner(48), [([("x", base[:300], [299]), ("y", other[:300], [299])], []),
                                         ([("x", base[300:], [0]), ("y", other[300:], [0])], ["x", "y"])])
    tm.check(tokens, got, "A far token")
    for position in (299, 300):
        want = tm.plain_logits(base)[position] - tm.plain_logits(other)[position]
        assert want.abs().max() > 1e-3
        assert pt.relative_error(got["x"][position] - got["y"][position], want) < 0.05


def test_sizes_come_from_the_configuration():
    """Values that a given model may leave equal to one another or at 1: one head, one kv head for many query heads, one
    tap on either side, a gate block of one channel and one block of all, a temperature that steps at every token, one
    expert, all experts chosen, a loop of one layer run once, a scale of 1, no cap."""
    one = pt.config(50, 32, 1e-3, 1.0, None, (1, 2, 1), [
        pt.layer(1, 1, 8, 4, 1, 6, 6, 1, pt.routed(8, 1, 1), temp=(2.0, 1), scale=1.0),
        pt.layer(5, 1, 8, 12, 5, 64, 1, 2, pt.routed(8, 3, 3, 0.3, (8, 5.0)), temp=None),
        pt.layer(2, 2, 4, 20, 2, 8, 2, 7, pt.dense(8, 0.2), temp=(0.01, 1000)),
        pt.layer(3, 3, 16, 12, 4, 40, 5, 4, None)])
    whole = pt.config(60, 24, 1e-6, 3.0, 20.0, (0, 3, 2), [
        pt.layer(2, 1, 16, 16, 2, 24, 2, 2, None), pt.layer(2, 2, 8, 16, 3, 16, 1, 3, pt.dense(20)),
        pt.layer(4, 2, 8, 8, 2, 12, 3, 4, pt.routed(12, 4, 2))])
    for cfg in (one, whole):
        for dtype in ("float32", "bfloat16"):
            tm = pt.TinyPakarax("-", dtype, cfg=cfg)
            tokens = {"p": pt.random_tokens(cfg, 40, 50)}
            steps = [([("p", tokens["p"][:20], list(range(20)))], [])]
            steps += [([("p", [t], [0])], []) for t in tokens["p"][20:]]
            tm.check(tokens, harness.replay(tm.runner(8), steps), "sizes of one")


def test_odd_sizes_and_a_larger_model():
    """A width that is no multiple of four with sizes that are no multiples of eight (every kernel's plain form), a model
    of wider rows, and rows wider than the tensor-core kernels take, under prompts, a second request and single
    tokens."""
    small = pt.config(101, 70, 1e-5, 1.3, 9.0, (0, 2, 2), [
        pt.layer(3, 3, 10, 6, 3, 35, 5, 2, pt.routed(30, 7, 3, 0.8, (18, 0.4))),
        pt.layer(6, 3, 14, 22, 2, 57, 3, 5, pt.dense(50)),
        pt.layer(9, 3, 22, 6, 4, 14, 2, 3, pt.routed(10, 9, 4))])
    large = pt.config(300, 200, 1e-6, 2.5, 15.0, (1, 3, 2), [
        pt.layer(8, 2, 80, 48, 4, 320, 4, 4, pt.routed(48, 12, 4, 0.9, (72, 0.8)), temp=(0.2, 100)),
        pt.layer(8, 4, 64, 24, 3, 256, 2, 4, pt.dense(352)),
        pt.layer(3, 1, 128, 96, 2, 144, 3, 2, pt.dense(352), temp=(0.3, 50)),
        pt.layer(8, 2, 48, 48, 4, 280, 1, 3, pt.routed(64, 8, 2))])
    wide = pt.config(90, 48, 1e-5, 1.0, 6.0, None, [
        pt.layer(2, 1, 160, 40, 3, 64, 2, 4, pt.dense(64), scale=0.1),
        pt.layer(4, 1, 40, 136, 2, 40, 1, 2, None)])
    for cfg, length in ((small, 120), (large, 450), (wide, 100)):
        for dtype in ("float32", "bfloat16"):
            tm = pt.TinyPakarax("-", dtype, cfg=cfg, seed=3)
            tokens = {"p": pt.random_tokens(cfg, length, 50), "q": pt.random_tokens(cfg, 77, 51)}
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

    width = pick([36, 52, 64, 100, 136])
    layers = []
    for _ in range(pick([2, 3, 4, 5])):
        kv = pick([1, 2, 3])
        dim = pick([8, 12, 16, 24, 32, 64])
        choice = pick(["none", "dense", "dense", "moe", "moe"])
        if choice == "none":
            mlp = None
        elif choice == "dense":
            mlp = pt.dense(pick([40, 72, 130]), pick([0.4, 1.0, 7.0]))
        else:
            experts = pick([1, 3, 8])
            mlp = pt.routed(pick([8, 24, 40]), experts, pick(list(range(1, experts + 1))), pick([0.4, 1.0, 7.0]),
                            pick([None, (16, 0.5), (48, 2.0)]))
        blocks = pick([1, 2, 3, 5])
        layers.append(pt.layer(kv * pick([1, 2, 3, 4]), kv, dim, pick([4, 8, 24, 64]), pick([1, 2, 3, 4, 5]),
                               blocks * pick([3, 8, 16, 20]), blocks, pick([1, 2, 3, 4, 6]), mlp,
                               temp=pick([None, (0.3, 1), (0.5, 13), (1.0, 64)]), scale=pick([0.1, 0.3, dim ** -0.5, 2 * dim ** -0.5])))
    start = pick(list(range(len(layers))))
    loop = pick([None, (start, pick(list(range(start + 1, len(layers) + 1))), pick([1, 2, 3]))])
    return pt.config(pick([64, 101, 257]), width, pick([1e-6, 1e-5, 1e-3]), pick([1.0, 0.5, 3.0]), pick([None, 4.0, 30.0]),
                     loop, layers)


@pytest.mark.parametrize("seed", list(range(12)))
def test_configurations_drawn_at_random(seed):
    """Each drawn model under a mixed schedule (portions, single tokens, a request that ends and one that takes its
    slot), float32 and bfloat16 against the plain implementation."""
    cfg = _random_config(seed)
    page = [16, 32, 64][seed % 3]
    for dtype in ("float32", "bfloat16"):
        tm = pt.TinyPakarax("-", dtype, seed=seed, cfg=cfg)
        tokens = {r: pt.random_tokens(cfg, n, 100 + seed + i) for i, (r, n) in enumerate({"a": 70, "b": 23, "c": 41}.items())}
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

    cfg, _ = pt.CONFIGS["A"]
    weights = pt.random_weights(cfg, 1)
    del weights["l2.mix.right.lam"]
    weights["l0.mix.left.sink"] = weights["l0.mix.left.sink"][:-1].contiguous()
    tm = pt.TinyPakarax("A", "float32", weights=weights)
    with pytest.raises((WeightsError, ValueError)) as error:
        load_model(tm.folder, "float32", DEV)
    assert "l2.mix.right.lam" in str(error.value) and "l0.mix.left.sink" in str(error.value)


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
    prompts = [pt.random_tokens(tm.cfg, n, 60 + i) for i, n in enumerate([40, 3, 21, 1, 30])]
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

    cfg, _ = pt.CONFIGS["B"]
    tm = pt.TinyPakarax("-", "float32", seed=4, cfg=cfg)
    engine = Engine(tm.folder, dtype="float32", device=DEV, page_size=16, n_pages=7, max_requests=4,
                    prefill_tokens_per_step=16)
    prompts = [pt.random_tokens(cfg, n, 95 + i) for i, n in enumerate([30, 25, 20])]
    requests = [engine.submit(p, max_tokens=20, ignore_eos=True) for p in prompts]
    for _ in range(600):
        if not engine.has_work():
            break
        engine.step()
    assert not engine.has_work() and engine.scheduler.preemptions > 0
    for prompt, request in zip(prompts, requests):
        assert request.finish_reason == "length"
        assert list(request.output) == _plain_greedy(tm, prompt, 20)


def test_captured_bfloat16_steps_equal_eager_ones():
    """Decode steps of several requests replayed from a capture (padding rows beside them) draw the tokens the eager
    steps draw, and their logits stay close to the plain implementation's."""
    from pulsarlm_b200.engine.engine import Engine

    tm = _model("C", "bfloat16")
    prompts = [pt.random_tokens(tm.cfg, n, 70 + i) for i, n in enumerate([50, 7, 33])]
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
                errors += [pt.relative_error(row, ref[len(prompt) - 1 + i]) for i, row in enumerate(request.logits)]
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
    assert "Pakarax" in capsys.readouterr().out.split()
    cfg, _ = pt.CONFIGS["C"]
    folder = str(tmp_path / "model")
    assert cli.main(["models", "random", folder, "--config", _write(tmp_path / "c.json", cfg), "--seed", "3",
                     "--dtype", "float32", "--std", "0.3"]) == 0
    capsys.readouterr()
    weights = {k: v.double() for k, v in load_file(folder + "/model.safetensors").items()}
    assert set(weights) == set(pt.tensor_shapes(cfg))
    prompt = pt.random_tokens(cfg, 19, 90)
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
    assert pt.relative_error(got0, ref[[3, 10]]) < 2e-4 and pt.relative_error(got2, ref[[11, 8]]) < 2e-4
    assert not (tmp_path / "out" / "1.f32").exists()
