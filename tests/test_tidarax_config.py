"""Tidarax: config.json -> configuration -> ModelSpec, random weights, and the plain implementation's own identities, on
the CPU."""

from __future__ import annotations

import copy
import math

import pytest
import torch

from jax_vllm_b200 import registry
from jax_vllm_b200.config.model_spec import RopeSpec
from jax_vllm_b200.models.tidarax import TidaraxConfig
from jax_vllm_b200.parts import BuildContext, Model
from jax_vllm_b200.parts.base import FixedStateNeed, PagedKVNeed
from jax_vllm_b200.parts.position import Rope
from jax_vllm_b200.weights.random_init import random_tensors
from tests.plain import tidarax_plain as tp
from tests.tidarax_util import CONFIGS, config, dense, layer, make_weights, moe, stored, tensor_shapes


def cpu_model(c):
    cfg = registry.config_from_dict(c)
    return cfg, Model(cfg.to_spec(), BuildContext(dtype=torch.float32, device=torch.device("cpu")))


@pytest.mark.parametrize("tag", sorted(CONFIGS))
def test_tensor_names_shapes_and_round_trip(tag):
    c = CONFIGS[tag]
    cfg, model = cpu_model(c)
    assert isinstance(cfg, TidaraxConfig)
    assert TidaraxConfig.from_dict(cfg.to_dict()) == cfg
    assert {k: tuple(v.shape) for k, v in model.tensor_specs().items()} == tensor_shapes(c)
    assert {k for k, v in model.tensor_specs().items() if v.kind == "table"} == {n for n in tensor_shapes(c) if n.endswith(".table")}


def test_what_every_layer_keeps_and_optional_norms():
    """Pages of keys and values (no wider for the mixed scores) and one state row; a folder may hold the second norm of a
    layer without a feed-forward."""
    c = CONFIGS["tb"]
    _, model = cpu_model(c)
    needs = model.cache_needs()
    assert needs[0] == (PagedKVNeed(3, 10, None, v_heads=3, v_head_dim=7), FixedStateNeed((33,), torch.float32))
    assert needs[2] == (PagedKVNeed(1, 20, None), FixedStateNeed((9,), torch.float32))
    assert "l0.norm2" in model.optional_tensors() and "l1.norm2" not in model.optional_tensors()


def test_random_weights_name_different_experts():
    c = config(70, 16, [layer(2, 1, 4, 4, 8, moe(7, 3, 8)), layer(2, 1, 4, 4, 8, moe(2, 2, 8))])
    _, model = cpu_model(c)
    w = random_tensors(model.tensor_specs(), 3, torch.float32)
    t = w["l0.mlp.table"]
    assert t.dtype == torch.int32 and t.shape == (70, 3) and int(t.min()) == 0 and int(t.max()) == 6
    assert all(len(set(row.tolist())) == 3 for row in t)
    assert sorted(w["l1.mlp.table"][0].tolist()) == [0, 1]
    assert (w["l0.mix.left.talk"] - torch.eye(2)).abs().max() < 0.8


@pytest.mark.parametrize("base,dims,scaling", [(1e4, 32, (8.0, 1.0, 4.0, 128.0)), (5e5, 64, (32.0, 2.0, 3.0, 8192.0)),
                                               (100.0, 6, (2.0, 1.0, 4.0, 40.0)), (1e4, 16, None)])
def test_frequencies_in_bands(base, dims, scaling):
    """The product's table against the plain function; with these constants every band holds at least one frequency."""
    spec = RopeSpec(dim=dims, theta=base, exact_table=True, bands=scaling)
    got = Rope(spec, "", BuildContext(dtype=torch.float32, device=torch.device("cpu"))).table()
    sc = None if scaling is None else dict(zip(("factor", "low", "high", "original"), scaling))
    want = tp.banded_frequencies(base, dims, sc)
    assert torch.allclose(got.double(), want, rtol=1e-7, atol=0.0)
    if scaling is not None:
        plain = tp.banded_frequencies(base, dims)
        ratio = (want / plain).tolist()
        assert ratio[0] == 1.0 and abs(ratio[-1] - 1.0 / scaling[0]) < 1e-12
        assert any(1.0 / scaling[0] + 1e-6 < r < 1.0 - 1e-6 for r in ratio)


def test_refusals():
    base = CONFIGS["ta"]

    def changed(f):
        c = copy.deepcopy(base)
        f(c)
        return c

    left = lambda c: c["layers"][0]["mixer"]["left"]
    for bad in (changed(lambda c: c["layers"][0].__setitem__("type", "unknown")),
                changed(lambda c: left(c).__setitem__("kv_heads", 4)),
                changed(lambda c: left(c)["rot"].__setitem__("dims", 7)),
                changed(lambda c: left(c)["rot"].__setitem__("dims", 18)),
                changed(lambda c: left(c)["rot"]["scaling"].pop("low")),
                changed(lambda c: c["layers"][0]["mixer"].pop("left_scale")),
                changed(lambda c: c["layers"][0]["mixer"]["right"].__setitem__("width", 0)),
                changed(lambda c: c["layers"][0]["mlp"].__setitem__("kind", "gated")),
                changed(lambda c: c["layers"][1]["mlp"]["router"].__setitem__("top", 6))):
        with pytest.raises((ValueError, KeyError)):
            registry.config_from_dict(bad)
    with pytest.raises(KeyError):
        registry.config_from_dict({k: v for k, v in base.items() if k != "norm"})


# ------------------------------------------------------------ the plain implementation's own identities
def test_plain_mixing_is_a_product_with_the_whole_key_row():
    """The mixed score of head h is one product of the whole key row with a query that holds, at each key head, the
    mixture of that key head's query heads."""
    g = torch.Generator().manual_seed(1)
    H, G, D, n = 6, 3, 5, 7
    q, k = (torch.randn((n, h, D), generator=g, dtype=torch.float64) for h in (H, G))
    T = torch.randn((H, H), generator=g, dtype=torch.float64)
    want = tp.talk(tp.raw_scores(q, k, 0.3), T)
    wide = torch.einsum("hcr,icrd->ihcd", T.view(H, G, H // G), q.view(n, G, H // G, D)).reshape(n, H, G * D)
    got = torch.einsum("ihx,jx->hij", wide, k.reshape(n, G * D)) * 0.3
    assert torch.allclose(got, want)
    # the identity mixes nothing, and a permutation of heads moves whole score maps
    assert torch.equal(tp.talk(want, torch.eye(H, dtype=torch.float64)), want)
    perm = torch.tensor([2, 0, 1, 5, 3, 4])
    assert torch.allclose(tp.talk(want, torch.eye(H, dtype=torch.float64)[perm]), want[perm])


def test_plain_zero_sink_and_unit_norm_after_rotation():
    g = torch.Generator().manual_seed(2)
    s = torch.randn((2, 4, 4), generator=g, dtype=torch.float64)
    w = tp.zero_sink_weights(s)
    e = torch.exp(s[1, 2, :3])
    assert torch.allclose(w[1, 2, :3], e / (1 + e.sum())) and float(w[1, 2, 3]) == 0.0
    assert tp.zero_sink_weights(s - 100.0).sum() < 1e-40                  # one is added whatever the scores
    assert tp.zero_sink_weights(s + 500.0)[0, 3].sum() > 1 - 1e-12         # and nothing overflows
    assert torch.allclose(tp.zero_sink_weights(s[:, 2:], first=2), w[:, 2:])
    x = torch.randn((5, 2, 8), generator=g, dtype=torch.float64)
    f = tp.banded_frequencies(100.0, 6)
    pos = torch.tensor([0, 3, 7, 50, 1])
    r = tp.rotate_halves(x, pos, f)
    assert torch.allclose(r[0], x[0]) and torch.allclose(r[..., 6:], x[..., 6:])
    assert torch.allclose(tp.unit(r, 1e-5), tp.rotate_halves(tp.unit(x, 1e-5), pos, f))    # a rotation keeps the mean square


def test_plain_recurrence_and_activation():
    g = torch.Generator().manual_seed(3)
    zl, y = (torch.randn((6, 4), generator=g, dtype=torch.float64) for _ in range(2))
    out, last = tp.gru_scan(zl, y)
    z, c = torch.sigmoid(zl), tp.candidate(y)
    for t in range(6):
        want = sum(z[s] * c[s] * torch.prod(1 - z[s + 1:t + 1], dim=0) for s in range(t + 1))
        assert torch.allclose(out[t], want)
    assert torch.allclose(tp.gru_scan(zl[3:], y[3:], tp.gru_scan(zl[:3], y[:3])[1])[1], last)
    assert float(tp.candidate(torch.tensor(0.0))) == 0.5 and abs(float(tp.candidate(torch.tensor(-1e-9, dtype=torch.float64))) - 0.5) < 1e-9
    v = torch.randn((3, 10), generator=g, dtype=torch.float64)
    coef = torch.tensor([1.5, -0.5, 0.25, 0.1], dtype=torch.float64)
    got = tp.poly_norm(v, coef, 1e-6)
    for t in range(3):
        rms = [math.sqrt(sum(float(x) ** (2 * k) for x in v[t]) / 10 + 1e-6) for k in (1, 2, 3)]
        for j in range(10):
            x = float(v[t, j])
            assert abs(float(got[t, j]) - (1.5 * x / rms[0] - 0.5 * x * x / rms[1] + 0.25 * x ** 3 / rms[2] + 0.1)) < 1e-12


def test_plain_table_of_experts():
    """Every token gets the mean of the experts its id's row names."""
    c = config(9, 6, [layer(1, 1, 4, 4, 3, moe(4, 2, 5))])
    w = stored(make_weights(c, 4))
    u = torch.randn((3, 6), generator=torch.Generator().manual_seed(5), dtype=torch.float64)
    tokens = [7, 2, 7]
    got = tp.table_ff(u, w, "l0.mlp", c["layers"][0]["mlp"], tokens)
    for t, tok in enumerate(tokens):
        a, b = w["l0.mlp.table"][tok].tolist()
        assert a != b
        want = 0.5 * (tp.expert(u[t:t + 1], w, f"l0.mlp.e{a}") + tp.expert(u[t:t + 1], w, f"l0.mlp.e{b}"))
        assert torch.allclose(got[t:t + 1], want)


def test_plain_forward_depends_on_earlier_tokens_only():
    c = config(30, 16, [layer(2, 1, 8, 6, 10, dense(12)), layer(2, 2, 4, 4, 5, moe(3, 2, 6))])
    w = stored(make_weights(c, 6))
    tokens = [3, 17, 4, 4, 29, 0, 11]
    full = tp.forward(c, w, tokens)
    assert torch.allclose(tp.forward(c, w, tokens[:4]), full[:4])
    other = tp.forward(c, w, tokens[:2] + [5] + tokens[3:])
    assert torch.allclose(other[:2], full[:2]) and (other[2:] - full[2:]).abs().min(dim=1).values.max() > 0
