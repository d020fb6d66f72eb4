"""The Pakarax decoder without a GPU: its configuration reader, its description as data, and the plain implementation's
own consistency."""

from __future__ import annotations

import json
import math

import pytest
import torch

import pakarax_tiny as pt
import plain_pakarax as plain

from pulsarlm_b200.config.base import ConfigError
from pulsarlm_b200.config.pakarax import PakaraxConfig
from pulsarlm_b200.config.registry import read_model_config, registered_architectures
from pulsarlm_b200.models.model import tensor_needs_of
from pulsarlm_b200.parts.filtered_attention import geometric_slopes, stacked_rows
from pulsarlm_b200.weights.loader import shape_fits


@pytest.mark.parametrize("key", ["A", "B", "C"])
def test_configuration_is_read_by_its_keys_and_written_back(key):
    text, _ = pt.CONFIGS[key]
    assert "Pakarax" in registered_architectures()
    arch, cfg = read_model_config(text)
    assert arch.name == "Pakarax" and isinstance(cfg, PakaraxConfig)
    assert PakaraxConfig.from_text(json.loads(json.dumps(cfg.to_text()))) == cfg
    for layer, entry in zip(cfg.layers, text["layers"]):
        a, r = entry["mixer"]["left"], entry["mixer"]["right"]
        left, right = layer.left, layer.right
        assert (left.heads, left.kv_heads, left.dim, left.vdim, left.taps) == tuple(
            a[n] for n in ("heads", "kv_heads", "dim", "vdim", "conv"))
        assert (right.width, right.blocks, right.taps) == (r["width"], r["blocks"], r["conv"])
        assert left.scale == a["scale"] and (layer.mlp is None) == (entry["mlp"] is None)
        assert (left.temp_coef, left.temp_every) == ((a["q_temp"]["coef"], a["q_temp"]["every"]) if "q_temp" in a
                                                      else (None, None))
    assert cfg.logit_scale == text["logit_scale"] and cfg.logit_softcap == text.get("logit_softcap")


@pytest.mark.parametrize("key", ["A", "B", "C"])
def test_described_model_needs_exactly_the_stored_tensors(key):
    text, _ = pt.CONFIGS[key]
    arch, cfg = read_model_config(text)
    spec = arch.describe(cfg)
    needs = tensor_needs_of(spec)
    shapes = pt.tensor_shapes(text)
    assert set(needs) == set(shapes)
    for name, shape in shapes.items():
        assert shape_fits(shape, needs[name].shape), name
    runs = plain.layer_runs(text)
    assert spec.order == [i for i, _ in runs] and list(spec.join_runs) == [r for r, (_, begins) in enumerate(runs) if begins]
    assert spec.cache_per_run


def test_a_key_left_out_takes_its_default():
    text = json.loads(json.dumps(pt.CONFIG_B))
    a = text["layers"][1]["mixer"]["left"]
    a.pop("kv_heads"), a.pop("vdim"), a.pop("q_temp"), text.pop("logit_scale")
    cfg = PakaraxConfig.from_text(text)
    left = cfg.layers[1].left
    assert left.kv_heads == left.heads and left.vdim == left.dim and left.temp_coef is None and cfg.logit_scale == 1.0
    assert cfg.runs() == ([0, 1, 2], [])


def test_bad_configurations_are_refused():
    for change in (lambda t: t["layers"][0].update(type="series"),
                   lambda t: t["layers"][1]["mixer"]["left"].update(kv_heads=4),
                   lambda t: t["layers"][0]["mixer"]["right"].update(blocks=5),
                   lambda t: t["layers"][0]["mixer"]["left"]["q_temp"].update(every=0),
                   lambda t: t["layers"][0]["mixer"]["left"].pop("scale"),
                   lambda t: t["layers"][0]["mlp"].pop("limit"),
                   lambda t: t["layers"][1]["mlp"]["router"].update(top=9),
                   lambda t: t["layers"][1]["mlp"].update(kind="sparse"),
                   lambda t: t["loop"].update(stop=4),
                   lambda t: t["loop"].update(times=0),
                   lambda t: t.pop("vocab")):
        bad = json.loads(json.dumps(pt.CONFIG_A))
        change(bad)
        with pytest.raises(ConfigError):
            PakaraxConfig.from_text(bad)


def test_slopes_and_stacked_operands():
    for heads in (1, 3, 8, 12):
        assert geometric_slopes(heads, 8.0) == plain.slopes(heads)
    assert geometric_slopes(8, 8.0)[0] == 0.5 and geometric_slopes(8, 8.0)[-1] == 2.0 ** -8
    parts = [torch.ones(5, 3), torch.full((8, 3), 2.0), torch.full((1, 3), 3.0)]
    whole, starts = stacked_rows(parts)
    assert starts == [0, 8, 16] and whole.shape == (24, 3)
    for part, at in zip(parts, starts):
        assert torch.equal(whole[at: at + part.shape[0]], part)
    assert float(whole[5:8].abs().sum()) == 0.0 == float(whole[17:].abs().sum())


def test_plain_implementation_is_causal_and_its_pieces_fit():
    cfg = pt.CONFIG_A
    weights = {k: v.double() for k, v in pt.random_weights(cfg, 2).items()}
    tokens = pt.random_tokens(cfg, 50, 1)
    whole = plain.forward(cfg, weights, tokens)
    assert plain.relative_error_of(plain.forward(cfg, weights, tokens[:31]), whole[:31]) < 1e-12
    assert float(whole.abs().max()) < cfg["logit_softcap"]
    # the recurrence cut in two with its state carried over
    gen = torch.Generator().manual_seed(3)
    u = torch.randn(20, 12, generator=gen).double()
    w = {"ra": torch.randn(3, 4, 4, generator=gen).double(), "ra.b": torch.randn(3, 4, generator=gen).double(),
         "ri": torch.randn(3, 4, 4, generator=gen).double(), "ri.b": torch.randn(3, 4, generator=gen).double(),
         "lam": torch.randn(12, generator=gen).double()}
    states = plain.linear_recurrence(u, w, 3)
    assert torch.allclose(plain.linear_recurrence(u[7:], w, 3, states[6]), states[7:])
    # a token alone sees itself and the sink; a sink of minus infinity is no sink
    q, k, v = torch.randn(9, 4, 8).double(), torch.randn(9, 2, 8).double(), torch.randn(9, 2, 6).double()
    none = torch.full((4,), float("-inf"), dtype=torch.float64)
    assert torch.equal(plain.sloped_attention(q, k, v, 0.3, none), plain.sloped_attention(q, k, v, 0.3, None))
    sink = torch.tensor([0.5, -1.0, 2.0, 0.0]).double()
    got = plain.sloped_attention(q, k, v, 0.3, sink)[0, 2]
    score = math.exp(0.3 * float(q[0, 2] @ k[0, 1]))
    assert torch.allclose(got, v[0, 1] * score / (score + math.exp(2.0)))
    # the temperature steps up at position every - 1 and starts at 1
    t = plain.query_temperature(torch.arange(12), 0.5, 4)
    assert [float(x) for x in t[:3]] == [1.0] * 3 and float(t[3]) == pytest.approx(1.0 + 0.5 * math.log(2.0))
    # the unit's limits: one-sided on the gate, two-sided on the other factor
    unit = plain.clamped_unit(torch.tensor([9.0, -9.0]).double(), torch.tensor([-9.0, 9.0]).double(), 2.0)
    assert float(unit[0]) == pytest.approx(2.0 / (1.0 + math.exp(-3.404)) * -1.0)
    assert float(unit[1]) == pytest.approx(-9.0 / (1.0 + math.exp(1.702 * 9.0)) * 3.0)
