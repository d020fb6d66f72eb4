"""The Zemarax decoder without a GPU: its configuration reader, its description as data, the cache that keeps a sequence's
first pages, and the plain implementation's own consistency."""

from __future__ import annotations

import json

import pytest
import torch

import plain_zemarax as plain
import zemarax_tiny as zt

from pulsarlm_b200.cache.manager import CacheManager, window_pages
from pulsarlm_b200.config.base import ConfigError
from pulsarlm_b200.config.registry import read_model_config, registered_architectures
from pulsarlm_b200.config.zemarax import ZemaraxConfig
from pulsarlm_b200.models.model import tensor_needs_of
from pulsarlm_b200.parts.spec import KVCacheNeed
from pulsarlm_b200.weights.loader import shape_fits


@pytest.mark.parametrize("key", ["A", "B", "C"])
def test_configuration_is_read_by_its_keys_and_written_back(key):
    text, _ = zt.CONFIGS[key]
    assert "Zemarax" in registered_architectures()
    arch, cfg = read_model_config(text)
    assert arch.name == "Zemarax" and isinstance(cfg, ZemaraxConfig)
    assert ZemaraxConfig.from_text(json.loads(json.dumps(cfg.to_text()))) == cfg
    for layer, entry in zip(cfg.layers, text["layers"]):
        m = entry["mixer"]
        assert (layer.mixer.heads, layer.mixer.dim, layer.mixer.vdim) == (m["heads"], m["dim"], m["vdim"])
        assert layer.mixer.window == (m.get("mask") or {}).get("size")
        assert layer.mixer.keep_first == (m.get("mask") or {}).get("keep_first", 0)
        assert layer.mixer.kv_from == m.get("kv_from") and (layer.mlp is None) == (entry["mlp"] is None)
    assert cfg.embedding_scale == text["embedding"]["scale"] and cfg.logit_scale == text["logit_scale"]


@pytest.mark.parametrize("key", ["A", "B", "C"])
def test_described_model_needs_exactly_the_stored_tensors(key):
    text, _ = zt.CONFIGS[key]
    arch, cfg = read_model_config(text)
    needs = tensor_needs_of(arch.describe(cfg))
    shapes = zt.tensor_shapes(text)
    assert {n for n, need in needs.items() if not need.optional} == set(shapes)
    for name, shape in shapes.items():
        assert shape_fits(shape, needs[name].shape), name


def test_bad_configurations_are_refused():
    text, _ = zt.CONFIGS["A"]
    for change in (lambda t: t["layers"][0].update(type="attention_9"),
                   lambda t: t["layers"][0]["mixer"].update(kv_heads=3),
                   lambda t: t["layers"][0]["mixer"]["mask"].update(size=0),
                   lambda t: t["layers"][0]["mixer"]["mask"].update(keep_first=-1),
                   lambda t: t["layers"][4]["mixer"].update(kv_from=1),      # (a layer of another kind)
                   lambda t: t["layers"][4]["mixer"].update(kv_from=4),      # (itself)
                   lambda t: t["layers"][4]["mixer"].update(kv_rank=16),     # (other latents than the source makes)
                   lambda t: t["layers"][1]["mixer"].update(gate_cap=0.0),
                   lambda t: t["layers"][0]["mlp"]["router"].update(top=9),
                   lambda t: t["layers"][1]["mlp"].update(kind="other"),
                   lambda t: t.pop("max_positions"), lambda t: t.pop("embedding")):
        bad = json.loads(json.dumps(text))
        change(bad)
        with pytest.raises(ConfigError):
            ZemaraxConfig.from_text(bad)


@pytest.mark.parametrize("keep,kept_pages", [(0, 0), (1, 1), (4, 1), (5, 2), (8, 2)])
def test_windowed_pages_go_back_and_the_first_ones_stay(keep, kept_pages):
    """Pages of 4, a window of 6: after every token the request holds the kept first pages and those the next query's
    window may reach; closing gives everything back."""
    cache = CacheManager([KVCacheNeed(1, 8, 6, 1, keep_first=keep), KVCacheNeed(1, 8, 6, 1)], 4, 64, 2, torch.float32, None,
                         allocate=False)
    assert len(cache.groups) == (1 if keep == 0 else 2)   # (layers that keep other tokens do not share pages)
    cache.open("r")
    for length in range(1, 60):
        assert cache.reserve("r", length)
        cache.commit("r", length)
        row = cache.table_rows(0, ["r"])[0]
        first = max(0, length - 6 + 1) // 4
        held = [i for i in range(-(-length // 4)) if row[i] >= 0]
        assert held == [i for i in range(-(-length // 4)) if i < kept_pages or i >= first], (length, held)
    cache.close("r")
    assert all(g["used"] == 0 for g in cache.stats()["groups"])
    assert window_pages(6, 4, 1, 3, keep) == window_pages(6, 4, 1, 3) + 3 * kept_pages


def test_plain_implementation_is_causal_and_its_pieces_fit():
    cfg, _ = zt.CONFIGS["A"]
    weights = {k: v.double() for k, v in zt.random_weights(cfg, 2).items()}
    tokens = zt.random_tokens(cfg, 60, 1)
    whole = plain.forward(cfg, weights, tokens)
    assert plain.relative_error_of(plain.forward(cfg, weights, tokens[:31]), whole[:31]) < 1e-12
    # reach: a window of the sequence's length is no window; kept tokens add to a window and never the future
    assert torch.equal(plain.in_reach(9, 9, 0), plain.in_reach(9, None, 0))
    seen = plain.in_reach(9, 2, 3)
    assert seen[8].tolist() == [True, True, True, False, False, False, False, True, True]
    assert seen[1].tolist() == [True, True] + [False] * 7
    # a sink far below every score is no sink; one far above leaves nothing
    q, k, v = torch.randn(9, 4, 8).double(), torch.randn(9, 2, 8).double(), torch.randn(9, 2, 6).double()
    full = plain.in_reach(9, None, 0)
    none = plain.sink_attention(q, k, v, 0.3, full, None)
    assert plain.relative_error_of(plain.sink_attention(q, k, v, 0.3, full, torch.full((4,), -60.0)), none) < 1e-12
    assert float(plain.sink_attention(q, k, v, 0.3, full, torch.full((4,), 60.0)).abs().max()) < 1e-12
    # the embedding: a portion that starts inside a sequence reads the token before it and its own positions
    table, pairs, places = (weights[n] for n in ("embed", "bigram", "pos"))
    both = plain.embedding(tokens, table, pairs, places, cfg)
    assert torch.equal(plain.embedding(tokens[20:], table, pairs, places, cfg, before=tokens[19], start=20), both[20:])
    # router weights: the softmax over the chosen logits alone
    h, router, bias = torch.randn(5, 16).double(), torch.randn(8, 16).double(), torch.randn(8).double()
    ids, w = plain.route(h, router, bias, 3)
    z = h @ router.T + bias
    for t in range(5):
        assert sorted(ids[t].tolist()) == sorted(z[t].topk(3).indices.tolist())
        assert torch.allclose(w[t], torch.softmax(z[t][ids[t]], 0))


def test_plain_matrix_memory_equals_its_unstabilised_form():
    """With gates small enough not to overflow, the stabilised recurrence equals the plain one: S' = sigmoid(f) S' +
    exp(i) k v^T, o = S'^T q / max(|n' q|, 1) (but for the 1e-6), and a portion continues where another stopped."""
    gen = torch.Generator().manual_seed(4)
    steps, heads, dim, vdim = 40, 3, 5, 7
    q, k = torch.randn(steps, heads, dim, generator=gen).double(), torch.randn(steps, heads, dim, generator=gen).double()
    v = torch.randn(steps, heads, vdim, generator=gen).double()
    i, f = plain.log_gates(torch.randn(steps, heads, generator=gen).double() * 3, torch.randn(steps, heads, generator=gen).double() + 2,
                           2.5)
    assert float(i.abs().max()) <= 2.5 and float(f.max()) < 0.0
    out, _ = plain.matrix_memory(q, k, v, i, f)
    s, n = torch.zeros(heads, dim, vdim).double(), torch.zeros(heads, dim).double()
    for t in range(steps):
        s = torch.exp(f[t])[:, None, None] * s + torch.exp(i[t])[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = torch.exp(f[t])[:, None] * n + torch.exp(i[t])[:, None] * k[t]
        want = torch.einsum("hd,hde->he", q[t], s) / (n * q[t]).sum(-1).abs().clamp(min=1.0)[:, None]
        assert plain.relative_error_of(out[t], want) < 1e-4, t
    first, state = plain.matrix_memory(q[:17], k[:17], v[:17], i[:17], f[:17])
    rest, _ = plain.matrix_memory(q[17:], k[17:], v[17:], i[17:], f[17:], state)
    assert torch.equal(torch.cat([first, rest]), out)


def test_stored_but_unused_norms_are_allowed_and_others_are_not():
    from pulsarlm_b200.weights.loader import WeightsError, check_names

    text, _ = zt.CONFIGS["A"]   # (its third layer has no feed-forward)
    arch, cfg = read_model_config(text)
    needs = tensor_needs_of(arch.describe(cfg))
    shapes = zt.tensor_shapes(text)
    shapes.update({"l2.norm2": (text["width"],), "l2.norm2b": (text["width"],)})
    check_names("a folder", needs, shapes)
    shapes["l4.mix.dkv"] = (32, text["width"])   # (a layer that reads another's latents makes none)
    with pytest.raises(WeightsError):
        check_names("a folder", needs, shapes)
