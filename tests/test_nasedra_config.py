"""Nasedra: config.json -> configuration -> ModelSpec, what its layers keep in the cache, and the plain implementation's own
identities, on the CPU."""

from __future__ import annotations

import copy
import math

import pytest
import torch

from jax_vllm_b200 import registry
from jax_vllm_b200.cache import CacheManager
from jax_vllm_b200.config.model_spec import RopeSpec
from jax_vllm_b200.models.nasedra import NasedraConfig
from jax_vllm_b200.parts import BuildContext, FixedStateNeed, Model, PagedKVNeed
from jax_vllm_b200.parts.position import Rope
from tests.nasedra_util import (CONFIGS, attention, config, dense, gla, layer, make_weights, moe, rotation, stored,
                                tensor_shapes)
from tests.plain import nasedra_plain as np_


def cpu_model(c):
    cfg = registry.config_from_dict(c)
    return cfg, Model(cfg.to_spec(), BuildContext(dtype=torch.float32, device=torch.device("cpu")))


@pytest.mark.parametrize("tag", sorted(CONFIGS))
def test_tensor_names_shapes_and_round_trip(tag):
    c = CONFIGS[tag]
    cfg, model = cpu_model(c)
    assert isinstance(cfg, NasedraConfig)
    assert NasedraConfig.from_dict(cfg.to_dict()) == cfg
    fit = lambda a, b: len(a) == len(b) and all(x in (-1, y) for x, y in zip(a, b))
    got, want = {k: tuple(v.shape) for k, v in model.tensor_specs().items()}, tensor_shapes(c)
    assert set(got) == set(want) and all(fit(got[k], want[k]) for k in got)


def test_what_every_layer_keeps():
    """Pages as wide as the widest mask among the owner and its readers, state rows, nothing for a reader; a folder may hold
    the second norm of a layer without a feed-forward."""
    _, model = cpu_model(CONFIGS["na"])
    needs = model.cache_needs()
    assert needs == [FixedStateNeed((3 * 12 * 20,), torch.float32),
                     PagedKVNeed(3, 16, 40, v_heads=3, v_head_dim=24, keep_first=6), FixedStateNeed((2 * 16 * 8,), torch.float32), None]
    assert "l3.norm2" in model.optional_tensors() and "l1.norm2" not in model.optional_tensors()
    _, model = cpu_model(CONFIGS["nb"])
    assert model.cache_needs()[0] == PagedKVNeed(1, 10, None, v_heads=1, v_head_dim=7)
    _, model = cpu_model(CONFIGS["nc"])
    assert model.cache_needs()[0] == PagedKVNeed(2, 64, None, v_heads=2, v_head_dim=80)      # a reader without a window
    assert model.cache_needs()[2] == PagedKVNeed(4, 32, 33)


def test_needs_of_owner_and_reader():
    win = lambda w, k=0: PagedKVNeed(2, 8, window=w, keep_first=k)
    chunk = lambda n: PagedKVNeed(2, 8, chunk=n)
    everything = PagedKVNeed(2, 8)
    assert win(5, 1).for_reader(win(9)) == win(9, 1) and win(9, 1).for_reader(win(5, 3)) == win(9, 3)
    assert win(5, 1).for_reader(everything) == everything and everything.for_reader(win(5, 1)) == everything
    assert chunk(8).for_reader(chunk(8)) == chunk(8) and chunk(8).for_reader(chunk(6)) == everything
    assert chunk(8).for_reader(win(5)) == everything


@pytest.mark.parametrize("keep", [1, 3, 4, 5, 9, 40])
def test_pages_of_kept_tokens_stay(keep):
    """As a request grows, exactly the pages that the next query can see stay, and release gives every one back; a new
    request with the same prefix finds the kept pages and the window's."""
    P, window = 4, 10
    m = CacheManager([PagedKVNeed(1, 8, window=window, keep_first=keep)], page_size=P, num_pages=40, max_live=2)
    rc = m.admit("a", list(range(70)))
    done = 0
    for n in (3, 1, 14, 2, 1, 1, 20, 6, 1, 21):
        m.grow(rc, done + n)
        m.commit(rc, list(range(done, done + n)))
        done += n
        m.check()
        held = {i for i in range(len(rc.tables[0])) if rc.tables[0][i] >= 0}
        needed = {j // P for j in range(done) if done - j < window or j < keep}
        assert held >= needed and all(i in needed or (i + 1) * P > done - window + 1 for i in held), (done, held, needed)
    rc2 = m.admit("b", list(range(70)))
    assert rc2.num_tokens == 68
    held = {i for i in range(17) if rc2.tables[0][i] >= 0}
    assert held == {j // P for j in range(68) if 68 - j < window or j < keep}
    m.check()
    m.release("a"); m.release("b")
    m.check()
    assert m.groups[0].pool.num_free == 40


@pytest.mark.parametrize("base,dims,scaling", [(1e4, 32, (8.0, 128.0, 4.0, 0.5)), (5e5, 64, (32.0, 8192.0, 32.0, 1.0)),
                                               (100.0, 6, (2.0, 40.0, 2.0, 1.0)), (1e3, 8, (1.0, 60.0, 4.0, 0.5)),
                                               (1e4, 16, (4.0, 10.0, 90.0, 80.0)), (1e4, 16, None)])
def test_yarn_frequencies(base, dims, scaling):
    """The product's table and gain against the plain function."""
    spec = RopeSpec(dim=dims, theta=base, exact_table=True, yarn=scaling, layout="interleaved")
    rope = Rope(spec, "", BuildContext(dtype=torch.float32, device=torch.device("cpu")))
    want, gain = np_.yarn_frequencies(base, dims, None if scaling is None else dict(zip(("factor", "original", "fast", "slow"), scaling)))
    assert torch.allclose(rope.table().double(), want, rtol=1e-7, atol=0.0) and abs(rope.gain - gain) < 1e-12


def test_yarn_by_hand():
    """Eight pairs, base 10^4, original 2 pi * 10^2: pair i turns 100 * 10^(-i/2) times, so d(t) = 2 log10(100 / t): fast =
    10 is pair 2, slow = 1 pair 4; pair 3 lies half way."""
    f, gain = np_.yarn_frequencies(1e4, 16, {"factor": 5.0, "original": 200.0 * math.pi, "fast": 10.0 * (1 - 1e-9), "slow": 1.0 + 1e-9})
    ratio = f / torch.tensor([10.0 ** (-i / 2) for i in range(8)], dtype=torch.float64)
    assert torch.allclose(ratio, torch.tensor([1.0, 1.0, 1.0, 0.6, 0.2, 0.2, 0.2, 0.2], dtype=torch.float64))
    assert abs(gain - (1.0 + 0.1 * math.log(5.0))) < 1e-12


def test_refusals():
    base = CONFIGS["na"]

    def changed(f):
        c = copy.deepcopy(base)
        f(c["layers"])
        return c

    mix = lambda ls, i: ls[i]["mixer"]
    for bad in (changed(lambda ls: ls[0].__setitem__("type", "unknown")),
                changed(lambda ls: mix(ls, 0).pop("tau")),
                changed(lambda ls: mix(ls, 0).__setitem__("tau", 0.0)),
                changed(lambda ls: mix(ls, 1).__setitem__("kv_heads", 4)),
                changed(lambda ls: mix(ls, 1)["rot"].__setitem__("dims", 7)),
                changed(lambda ls: mix(ls, 1)["rot"]["scaling"].pop("slow")),
                changed(lambda ls: mix(ls, 1).__setitem__("softcap", 0.0)),
                changed(lambda ls: mix(ls, 1)["mask"].__setitem__("size", 0)),
                changed(lambda ls: mix(ls, 3).__setitem__("kv_from", 0)),
                changed(lambda ls: mix(ls, 3).__setitem__("kv_from", 3)),
                changed(lambda ls: mix(ls, 3).__setitem__("vdim", 16)),
                changed(lambda ls: ls[0]["mlp"].__setitem__("kind", "gated")),
                changed(lambda ls: ls[1]["mlp"]["router"].__setitem__("top", 8)),
                changed(lambda ls: ls[1]["mlp"]["shared"].__setitem__("ff", 0))):
        with pytest.raises((ValueError, KeyError)):
            registry.config_from_dict(bad)
    for key in ("embedding", "norm", "width"):
        with pytest.raises(KeyError):
            registry.config_from_dict({k: v for k, v in base.items() if k != key})


# ------------------------------------------------------------ the plain implementation's own identities
def test_plain_visibility():
    see = np_.visible(9, window=3, keep_first=2)
    for i in range(9):
        assert [j for j in range(9) if see[i, j]] == sorted({j for j in range(i + 1) if i - j < 3} | {j for j in (0, 1) if j <= i})
    assert torch.equal(np_.visible(9, window=3, keep_first=2, first=5), see[5:])
    assert torch.equal(np_.visible(6), torch.ones(6, 6).tril().bool())


def test_plain_rotation_turns_neighbours():
    g = torch.Generator().manual_seed(1)
    x = torch.randn((4, 2, 8), generator=g, dtype=torch.float64)
    f = torch.tensor([1.0, 0.1, 0.01], dtype=torch.float64)
    pos = torch.tensor([0, 3, 7, 50])
    r = np_.rotate_pairs(x, pos, f, 1.3)
    z = torch.complex(x[..., 0:6:2], x[..., 1:6:2]) * 1.3 * torch.exp(1j * pos[:, None, None] * f)
    assert torch.allclose(r[..., 0:6:2], z.real) and torch.allclose(r[..., 1:6:2], z.imag) and torch.equal(r[..., 6:], x[..., 6:])


def test_plain_linear_attention_is_a_weighted_sum_of_values():
    g = torch.Generator().manual_seed(2)
    T, H, D, E = 6, 2, 3, 4
    q, k = (torch.randn((T, H, D), generator=g, dtype=torch.float64) for _ in range(2))
    v, z = torch.randn((T, H, E), generator=g, dtype=torch.float64), torch.randn((T, H, D), generator=g, dtype=torch.float64)
    a = np_.channel_decay(z, 4.0)
    assert torch.allclose(a, torch.sigmoid(z) ** 0.25)
    o, last = np_.gla_scan(q, k, v, a)
    for t in range(T):
        want = sum((q[t] * k[s] * torch.prod(a[s + 1:t + 1], dim=0)).sum(-1, keepdim=True) * v[s] for s in range(t + 1))
        assert torch.allclose(o[t], want)
    o1, S = np_.gla_scan(q[:4], k[:4], v[:4], a[:4])
    assert torch.allclose(np_.gla_scan(q[4:], k[4:], v[4:], a[4:], S)[1], last)


def test_plain_router_with_correction_and_identity_experts():
    """The correction decides who is chosen and never how much; identity experts give the token itself."""
    c = config(9, 6, [layer(gla(1, 2, 2, 1.0), moe(2, 2, 5, identity=2, scale=3.0))])
    w = stored(make_weights(c, 4))
    ml = c["layers"][0]["mlp"]
    u = torch.randn((5, 6), generator=torch.Generator().manual_seed(5), dtype=torch.float64)
    w["l0.mlp.correction"] = torch.tensor([-5.0, 5.0, -5.0, 5.0], dtype=torch.float64)
    s = torch.softmax(u @ w["l0.mlp.router"].T, dim=-1)
    total = s[:, 1:2] + s[:, 3:4]
    want = 3.0 * (s[:, 1:2] * np_.gated(u, w, "l0.mlp.e1") + s[:, 3:4] * u) / total
    assert torch.allclose(np_.moe(u, w, "l0.mlp", ml), want)


def test_plain_forward_depends_on_earlier_tokens_only():
    c = config(30, 16, [layer(gla(2, 4, 3, 2.0), dense(12)), layer(attention(2, 1, 8, 6, rotation(4), size=3, keep=1, cap=4.0), moe(3, 2, 6, 1)),
                        layer(attention(2, 1, 8, 6, rotation(4), kv_from=1), None)])
    w = stored(make_weights(c, 6))
    tokens = [3, 17, 4, 4, 29, 0, 11]
    full = np_.forward(c, w, tokens)
    assert torch.allclose(np_.forward(c, w, tokens[:4]), full[:4])
    other = np_.forward(c, w, tokens[:2] + [5] + tokens[3:])
    assert torch.allclose(other[:2], full[:2]) and (other[2:] - full[2:]).abs().max(dim=1).values.min() > 0
