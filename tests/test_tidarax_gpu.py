"""The Tidarax design in the engine against the plain implementation (tests/plain/tidarax_plain.py): every mechanism
alone, then models of several sizes through the replay program's class (whole, last tokens one by one, portions down to
two tokens, unequal requests side by side in reused pages and state slots), special weights where random ones would hide
a fault, and greedy generation through the entry point and its scheduler."""

from __future__ import annotations

import json
import math
import os
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from tests.plain import tidarax_plain as tp
from tests.test_nufapel_gpu import mixed_trace, scrambled_pages
from tests.test_replay_gpu import limits
from tests.tidarax_util import CONFIGS, PAGE, config, dense, layer, make_weights, moe, rotation, stored, write_folder
from tests.util import collect, portions, prefix_then_single, random_tokens, whole

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
LENGTHS = {"ta": [70, 45, 100, 33, 52], "tb": [90, 38, 64, 51, 27], "tc": [200, 70, 150, 40, 66], "td": [61, 40, 83, 35, 20],
           "te": [310, 60, 140, 37, 45]}


def oracle(c, w, tokens):
    return tp.forward(c, w, tokens).to(torch.float32)


def rounding_error(c, w, tokens):
    """Per position, how far the plain logits move when the operands and the result of every matrix product are rounded to
    bfloat16 and nothing else is: what rounding alone does to this model at this token."""
    bf = lambda x: x.to(torch.bfloat16).to(torch.float64)
    exact = tp.forward(c, w, tokens)
    plain_matmul = torch.Tensor.__matmul__
    torch.Tensor.__matmul__ = lambda a, b: bf(plain_matmul(bf(a), bf(b)))
    try:
        rounded = tp.forward(c, w, tokens)
    finally:
        torch.Tensor.__matmul__ = plain_matmul
    return (rounded - exact).abs().max(dim=1).values


def compare(steps, out_dir, vocab, want, dtype, case=None, rounding=None):
    """Every written row against the oracle's.  32-bit holds every position and the greedy token.  In bfloat16 one
    position in fifty (or one) may be over the limit by up to half of it.  `rounding` (request -> `rounding_error`): a
    bfloat16 position's limit is at least three times what rounding alone does there, for models drawn at random."""
    from tests.conftest import record_worst
    got = collect(steps, out_dir, vocab)
    worst, lim_of_worst, total, slightly = 0.0, 0.0, 0, 0
    for rid, rows in got.items():
        lim_all = limits(dtype, want[rid])
        for pos, row in rows.items():
            total += 1
            lim = lim_all
            if rounding is not None and dtype != "float32":
                lim = max(lim, 3.0 * float(rounding[rid][pos]))
            w = want[rid][pos]
            diff = (torch.from_numpy(row.copy()) - w).abs().max().item()
            assert math.isfinite(diff), f"{rid} position {pos}: not a number"
            if dtype != "float32" and lim < diff <= 1.5 * lim:
                slightly += 1
                continue
            assert diff <= lim, f"{rid} position {pos}: |diff| {diff:.3e} > {lim:.3e}"
            if diff >= worst:
                worst, lim_of_worst = diff, lim
            if dtype == "float32":
                top2 = w.topk(2).values
                assert int(row.argmax()) == int(w.argmax()) or float(top2[0] - top2[1]) < 1e-4
    share = 0.1 if rounding is not None else 0.02
    assert slightly <= max(1, share * total), f"{slightly} of {total} positions are over the limit"
    if case is not None:
        record_worst(case, dtype, worst, lim_of_worst)
    return got


@pytest.fixture(scope="module", params=sorted(CONFIGS))
def setup(request, tmp_path_factory):
    tag = request.param
    c = CONFIGS[tag]
    weights = make_weights(c, seed=5)
    folder = write_folder(tmp_path_factory.mktemp(f"tidarax_{tag}"), c, weights)
    w = stored(weights)
    seqs = {f"r{i}": random_tokens(n, c["vocab"], seed=20 + i) for i, n in enumerate(LENGTHS[tag])}
    want = {rid: oracle(c, w, t) for rid, t in seqs.items()}
    assert all(v.abs().max() > 1.0 for v in want.values())     # logits of order one, not a flat model
    return tag, folder, seqs, want


def replay(folder, tag, dtype, steps, out_dir, max_tokens, **switches):
    from jax_vllm_b200.engine.replay import Replayer
    rep = Replayer(folder, dtype, out_dir, max_tokens=max_tokens, page_size=PAGE[tag], **switches)
    rep.run_stream(json.dumps(s) for s in steps)
    rep.cache.check()
    assert not rep.cache.live
    return rep


def entries_of(lengths, slots):
    cu = torch.tensor([0] + list(torch.tensor(lengths).cumsum(0)), dtype=torch.int32).cuda()
    return cu, torch.tensor(slots, dtype=torch.int32).cuda()


def step_of(ctx_new, table, tile_classes, slots=None, tokens=None):
    """A step context for entries of (cached, new) tokens, as the engine's batch builder lays it out."""
    from jax_vllm_b200.parts.base import StepContext
    lengths = [q for _, q in ctx_new]
    n = sum(lengths)
    cu, sl = entries_of(lengths, slots if slots is not None else list(range(len(ctx_new))))
    i32 = lambda x: torch.tensor(x, dtype=torch.int32).cuda()
    work = {}
    for tpt, lo, hi in tile_classes:
        lst = [(e, t) for e, (_, q) in enumerate(ctx_new) if q > 1 and lo <= q < hi for t in range(0, q, tpt)]
        work[(tpt, lo, hi)] = (i32(lst).view(-1, 2), len(lst))
    singles = [(e, 0) for e, (_, q) in enumerate(ctx_new) if q == 1]
    return StepContext(n_tokens=n, n_entries=len(ctx_new), token_ids=i32(tokens if tokens is not None else [0] * n),
                       positions=i32([p for c, q in ctx_new for p in range(c, c + q)]),
                       token_entry=i32([e for e, (_, q) in enumerate(ctx_new) for _ in range(q)]), cu_seqlens=cu,
                       start_pos=i32([c for c, _ in ctx_new]), state_slots=sl, logit_rows=i32([]), n_logit_rows=0,
                       block_tables=[table.cuda()] if table is not None else [], tile_work=work,
                       decode_work=(i32(singles).view(-1, 2), len(singles)), max_seq_len=max(c + q for c, q in ctx_new))


# ------------------------------------------------------------------ mechanisms alone
# (query heads, key heads, key size, value size, rotated elements)
PREPARE_CASES = [(6, 3, 16, 8, 8), (3, 1, 21, 12, 20), (4, 4, 32, 64, 0), (1, 1, 70, 34, 40), (16, 1, 12, 4, 12),
                 (16, 4, 128, 128, 128), (32, 8, 128, 64, 64), (5, 5, 7, 3, 2)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,E,rot", PREPARE_CASES)
@pytest.mark.parametrize("tokens", ["several", "many"])
def test_mixed_queries_alone(H, G, D, E, rot, tokens, dtype):
    """Rotation in halves with banded frequencies, unit norm per head, the mixture of query heads at every key head's
    place, keys and values into scrambled pages; a few tokens (several blocks a token) and many (one)."""
    from jax_vllm_b200 import ops
    g = torch.Generator().manual_seed(H * D + E)
    P, n_pages, eps = 8, 60, 1e-4
    ctx_new = [(37, 21), (0, 3), (130, 1)] if tokens == "several" else [(5, 160), (0, 30)]
    table = scrambled_pages(ctx_new, P, n_pages, g)
    n = sum(q for _, q in ctx_new)
    pos = torch.cat([torch.arange(c, c + q) for c, q in ctx_new])
    ent = torch.cat([torch.full((q,), e) for e, (_, q) in enumerate(ctx_new)])
    cols = H * D + G * D + G * E
    proj = (1.5 * torch.randn((n, cols + 3), generator=g)).to(dtype)
    T = (torch.eye(H) + 0.7 * torch.randn((H, H), generator=g))
    freq = tp.banded_frequencies(5e3, rot, dict(factor=4.0, low=1.0, high=4.0, original=50)).float() if rot else None
    kc = torch.zeros((n_pages, P, G, D), dtype=dtype).cuda()
    vc = torch.zeros((n_pages, P, G, E), dtype=dtype).cuda()
    q_out = torch.full((n, H * G * D), float("nan"), dtype=dtype).cuda()
    ops.talk_prepare(proj.cuda(), 3, 3 + H * D, 3 + H * D + G * D, q_out, T.cuda(), pos.int().cuda(), ent.int().cuda(),
                     table.cuda(), None if freq is None else freq.cuda(), eps, kc, vc, H, G, D, E)
    ops.check_status()
    x = proj.double()
    q, k = x[:, 3:3 + H * D].view(n, H, D), x[:, 3 + H * D:3 + H * D + G * D].view(n, G, D)
    v = x[:, 3 + H * D + G * D:3 + cols].view(n, G, E)
    if freq is not None:
        q, k = tp.rotate_halves(q, pos, freq.double()), tp.rotate_halves(k, pos, freq.double())
    q, k = tp.unit(q, eps), tp.unit(k, eps)
    wide = torch.einsum("hcr,icrd->ihcd", T.double().view(H, G, H // G), q.view(n, G, H // G, D)).reshape(n, H * G * D)
    tol = 3e-5 if dtype == torch.float32 else 1e-2
    close = lambda a, b: (a.double().cpu() - b).abs().max().item() < tol * max(1.0, b.abs().max().item())
    assert close(q_out, wide)
    for t in range(n):
        page, slot = int(table[ent[t], pos[t] // P]), int(pos[t] % P)
        assert close(kc[page, slot], k[t]) and torch.equal(vc[page, slot].double().cpu(), v[t]), t


# name: (query heads, key heads, key size, value size, what serves it in bfloat16)
TALK_CASES = {"general_96x48": (4, 2, 48, 48), "general_256x32": (8, 8, 32, 32), "general_16x64": (1, 1, 16, 64),
              "general_512x64": (16, 8, 64, 64), "general_384x128": (6, 6, 64, 128), "many_heads": (96, 6, 32, 32),
              "odd_sizes": (3, 3, 21, 7), "wide_rows": (4, 4, 96, 40), "very_wide_rows": (12, 12, 130, 20),
              "one_key_head": (16, 1, 64, 32), "heads_of_128_on_2": (4, 2, 128, 128), "heads_of_128_on_4": (8, 4, 128, 128),
              "heads_of_128_on_8": (8, 8, 128, 128), "heads_of_128_on_1": (3, 1, 128, 128),
              "many_heads_of_128_on_4": (32, 4, 128, 128)}


def talking_part(H, G, D, E, scale, dtype, rot, eps, out_scale, T):
    from jax_vllm_b200.config.model_spec import GeneralAttentionSpec, RopeSpec
    from jax_vllm_b200.parts import BuildContext
    from jax_vllm_b200.parts.general_attention import GeneralAttention
    spec = GeneralAttentionSpec(hidden_size=8, num_heads=H, num_kv_heads=G, key_dim=D, value_dim=E, scale=scale,
                                position=RopeSpec(dim=rot, theta=1e4, exact_table=True) if rot else None, head_norm_eps=eps,
                                head_norm_weight=False, talk=True, sink_score=0.0, output_scale=out_scale, prefix="m")
    part = GeneralAttention(spec, "l", BuildContext(dtype, torch.device("cuda"), decode_split_size=64))
    zeros = {k: torch.zeros(v.shape, device="cuda", dtype=torch.bfloat16) for k, v in part.tensor_specs().items()}
    part.bind({**zeros, "l.m.talk": T.cuda()})
    return part


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", sorted(TALK_CASES))
def test_attention_with_mixed_scores_alone(name, dtype):
    """From a projection to the heads: a prompt portion over several tiles behind earlier context, a short portion of two
    tokens, a prompt from position 0, and single tokens whose keys are split into ranges (one of them the first token of
    its sequence), in one batch over scrambled pages; scores spread enough that the weights are sharp; the mixing and the
    added one matter (without either the plain result differs by far more than the limit)."""
    from jax_vllm_b200 import ops
    from jax_vllm_b200.parts.base import PagedLayerCache
    H, G, D, E = TALK_CASES[name]
    g = torch.Generator().manual_seed(H * D + E)
    P, n_pages, eps, rot, out_scale = 16, 64, 1e-5, (D // 4) * 2, 0.7
    scale = 2.0 * D ** -0.5
    T = torch.eye(H) + (0.6 / H ** 0.5) * torch.randn((H, H), generator=g)
    part = talking_part(H, G, D, E, scale, dtype, rot, eps, out_scale, T)
    ctx_new = [(37, 145), (70, 2), (0, 3), (200, 1), (0, 1)]
    table = scrambled_pages(ctx_new, P, n_pages, g)
    step = step_of(ctx_new, table, part.tile_classes(P))
    n, cols = step.n_tokens, part.in_rows
    full = [torch.randn((c + q, cols), generator=g).to(dtype) for c, q in ctx_new]          # projections of whole sequences
    freq = tp.banded_frequencies(1e4, rot)
    kc = torch.full((n_pages, P, G, D), float("nan"), dtype=dtype)
    vc = torch.full((n_pages, P, G, E), float("nan"), dtype=dtype)
    want, bare, unmixed = [], [], []
    for e, (c, q) in enumerate(ctx_new):
        x = full[e].double()
        qq, kk, vv = x[:, :H * D].view(-1, H, D), x[:, H * D:(H + G) * D].view(-1, G, D), x[:, (H + G) * D:].view(-1, G, E)
        pos = torch.arange(c + q)
        qq, kk = (tp.unit(tp.rotate_halves(y, pos, freq), eps) for y in (qq, kk))
        for j in range(c):                                                                  # what earlier steps left
            kc[table[e, j // P], j % P], vc[table[e, j // P], j % P] = kk[j].to(dtype), vv[j].to(dtype)
        want.append(out_scale * tp.talking_attend(qq[c:], kk, vv, scale, T.double(), first=c))
        unmixed.append(out_scale * tp.talking_attend(qq[c:], kk, vv, scale, torch.eye(H, dtype=torch.float64), first=c))
        s = tp.talk(tp.raw_scores(qq[c:], kk, scale), T.double())
        s = s.masked_fill(torch.arange(c + q)[None, :] > (c + torch.arange(q))[:, None], -math.inf)
        bare.append(out_scale * torch.einsum("hij,jhe->ihe", s.softmax(-1), vv.repeat_interleave(H // G, dim=1)))
    rows = torch.cat([full[e][c:] for e, (c, _) in enumerate(ctx_new)]).cuda()
    wide = torch.full((n, H * E + 8), float("nan"), dtype=dtype).cuda()
    part.from_projection(rows, step, PagedLayerCache(0, kc.cuda(), vc.cuda()), wide[:, :H * E])
    ops.check_status()
    assert bool(torch.isnan(wide[:, H * E:]).all())
    got = wide[:, :H * E].cpu().double().view(n, H, E)
    tol = 3e-5 if dtype == torch.float32 else 3e-2
    at = 0
    for e, (c, q) in enumerate(ctx_new):
        size = max(1.0, want[e].abs().max().item())
        assert (got[at:at + q] - want[e]).abs().max() < tol * size, f"entry {e}: {(got[at:at + q] - want[e]).abs().max()}"
        at += q
    moved = lambda others: max((o - w).abs().max().item() for o, w in zip(others, want))
    assert moved(bare) > 0.1 and (H == 1 or moved(unmixed) > 0.1)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("C", [1, 16, 33, 200, 4096])
def test_recurrence_alone(C, dtype):
    """Entries of unequal length (one over several tiles of tokens, one of a single token, one at a tile's edge) whose
    states lie in slots given out of order; a second call carries on from what the first left; single tokens alone; an
    unused slot stays as it was.  Gates far on both sides of zero; input and output are column ranges."""
    from jax_vllm_b200 import ops
    g = torch.Generator().manual_seed(C)
    first, second, third, slots, n_slots = [1300, 1, 1537, 9], [1, 3, 260, 1], [1, 1, 1, 1], [3, 0, 4, 1], 6
    zb, xb = (torch.randn(C, generator=g).to(dtype) for _ in range(2))
    total = [a + b + c for a, b, c in zip(first, second, third)]
    full = [(3.0 * torch.randn((t, 3 * C), generator=g)).to(dtype) for t in total]
    full[0][:, 0] = -9.0                                       # a channel that hardly ever lets anything in
    full[2][5:9, :C] = 90.0                                    # gates that take the candidate whole
    full[2][20:25, :C] = -90.0
    start = [torch.randn(C, generator=g) for _ in total]
    state = torch.full((n_slots, C + 2), 7.0)
    for e, s in enumerate(slots):
        state[s, :C] = start[e]
    state = state.cuda()
    want = [tp.gru_scan(f[:, :C].double() + zb.double(), f[:, C:2 * C].double() + xb.double(), s.double())
            for f, s in zip(full, start)]
    done = [0] * 4
    for lengths in (first, second, third):
        rows = torch.cat([full[e][done[e]:done[e] + n] for e, n in enumerate(lengths)])
        wide = torch.cat([torch.full((rows.shape[0], 5), float("nan")), rows.float()], 1).to(dtype).cuda()
        cu, sl = entries_of(lengths, slots)
        out = torch.full((rows.shape[0], C + 3), float("nan"), dtype=dtype).cuda()
        ops.min_gru(wide, 5, 5 + C, 5 + 2 * C, zb.cuda(), xb.cuda(), state[:, :C], cu, sl, 4, C, out[:, 3:], scale=0.6)
        ops.check_status()
        assert bool(torch.isnan(out[:, :3]).all())
        at = 0
        for e, n in enumerate(lengths):
            S = want[e][0][done[e]:done[e] + n]
            ref = 0.6 * S * tp.silu(full[e][done[e]:done[e] + n, 2 * C:].double())
            tol = 1e-5 if dtype == torch.float32 else 8e-3
            err = (out[at:at + n, 3:].double().cpu() - ref).abs() / torch.clamp(ref.abs(), min=1.0)
            assert err.max() < tol, (e, lengths)
            at += n
            done[e] += n
            left = state[slots[e], :C].double().cpu()
            assert ((left - want[e][0][done[e] - 1]).abs() / torch.clamp(left.abs(), min=1.0)).max() < 1e-5, (e, lengths)
    assert bool((state[2] == 7.0).all() and (state[5] == 7.0).all() and (state[:, C:] == 7.0).all())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,width", [(1, 4), (3, 33), (2, 1000), (200, 512), (5, 12288), (150, 16384), (2, 40000)])
def test_activation_of_normed_powers_alone(n, width, dtype):
    """As a tensor, as a column range, and as the parts of a sum."""
    from jax_vllm_b200 import ops
    g = torch.Generator().manual_seed(n + width)
    z = torch.randn((n, width), generator=g).to(dtype)
    z[0] = 0.0 if n > 1 else z[0]                              # a row of zeros: only eps stands in the roots
    coef = torch.tensor([1.2, -0.7, 0.4, 0.3]).to(dtype)
    want = tp.poly_norm(z.double(), coef.double(), 1e-5)
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    close = lambda a: ((a.double().cpu() - want).abs() / torch.clamp(want.abs(), min=1.0)).max().item() < tol
    assert close(ops.poly_norm(z.cuda(), coef.cuda(), 1e-5))
    wide = torch.full((n, width + 9), float("nan"), dtype=dtype)
    wide[:, 4:4 + width] = z
    out = torch.full((n, width + 9), float("nan"), dtype=dtype).cuda()
    ops.poly_norm(wide.cuda()[:, 4:4 + width], coef.cuda(), 1e-5, out=out[:, 8:8 + width])
    assert close(out[:, 8:8 + width]) and bool(torch.isnan(out[:, :8]).all())
    parts = torch.randn((3, n, width), generator=g)
    parts[2] = z.float() - parts[0] - parts[1]
    got = ops.poly_norm(ops.PartialSum(parts.cuda()), coef.cuda(), 1e-5, out_dtype=dtype)
    if n == 1:
        assert close(got)
    else:
        err = ((got.double().cpu() - want).abs() / torch.clamp(want.abs(), min=1.0))[1:]
        assert err.max() < max(tol, 1e-4)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("E,top,F,W,n", [(5, 3, 24, 40, 33), (1, 1, 8, 16, 5), (8, 2, 128, 128, 150), (4, 4, 136, 256, 1), (64, 6, 128, 256, 300)])
def test_experts_named_by_a_table_alone(E, top, F, W, n, dtype):
    """Gated silu experts chosen by token id, on the CUDA-core and the tensor-core grouped products."""
    from jax_vllm_b200 import ops
    from jax_vllm_b200.config.model_spec import RoutedExpertsSpec
    from jax_vllm_b200.parts import BuildContext
    from jax_vllm_b200.parts.routed_experts import RoutedExperts
    vocab = 50
    c = config(vocab, W, [layer(1, 1, 4, 4, 3, moe(E, top, F))])
    w = {k[3:]: v for k, v in make_weights(c, 7).items() if k.startswith("l0.mlp")}
    part = RoutedExperts(RoutedExpertsSpec(W, E, top, F, scoring="table", activation="swiglu", vocab_size=vocab), "",
                         BuildContext(dtype, torch.device("cuda")))
    part.prefix = "mlp"
    part.bind({k: (v.to(torch.bfloat16) if v.is_floating_point() else v).cuda() for k, v in w.items()})
    tokens = random_tokens(n, vocab, 3)
    x = torch.randn((n, W), generator=torch.Generator().manual_seed(2)).to(dtype)
    got = part.forward(x.cuda(), step_of([(0, n)], None, [], tokens=tokens)).tensor().double().cpu()
    ops.check_status()
    want = tp.table_ff(x.double(), stored(w), "mlp", c["layers"][0]["mlp"], tokens)
    tol = 2e-5 if dtype == torch.float32 else 3e-2
    assert (got - want).abs().max() < tol * max(1.0, want.abs().max().item())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,hidden,top", [(5, 40, 1), (7, 33, 3), (200, 2048, 4), (3, 8192, 9)])
def test_a_norm_that_picks_up_the_experts_rows(n, hidden, top, dtype):
    """The sum of weighted rows added and normed in one pass, for all rows (the stream is updated) and for chosen rows (it
    is not), against the two steps apart."""
    from jax_vllm_b200 import ops
    g = torch.Generator().manual_seed(n + hidden)
    h = torch.randn((n, hidden), generator=g)
    rows = torch.randn((2 * n + 3, hidden), generator=g).to(dtype)
    pick = torch.randint(0, 2 * n + 3, (n, top), generator=g, dtype=torch.int32)
    coef = torch.randn((n, top), generator=g)
    w = (1.0 + 0.1 * torch.randn(hidden, generator=g)).to(dtype)
    full = h.double() + torch.einsum("ns,nsc->nc", coef.double(), rows.double()[pick.long()])
    want = tp.unit(full, 1e-5) * w.double()
    hc = h.cuda()
    delta = ops.PickedRows(rows.cuda(), pick.cuda(), coef.cuda())
    some = torch.tensor([n - 1, 0, n // 2], dtype=torch.int32)
    y = ops.rmsnorm(hc, w.cuda(), 1e-5, dtype, delta=delta, rows=some.cuda())
    assert torch.equal(hc.cpu(), h)
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    assert (y.double().cpu() - want[some.long()]).abs().max() < tol * want.abs().max()
    y = ops.rmsnorm(hc, w.cuda(), 1e-5, dtype, delta=delta)
    ops.check_status()
    assert (y.double().cpu() - want).abs().max() < tol * want.abs().max()
    assert (hc.double().cpu() - full).abs().max() < 1e-5 * full.abs().max()


def test_a_table_that_names_no_expert_is_reported():
    from jax_vllm_b200 import ops
    table = torch.tensor([[0, 1], [2, 5]], dtype=torch.int32).cuda()
    ids, wt = ops.moe_route_table(torch.tensor([0, 1], dtype=torch.int32).cuda(), table, 4)
    with pytest.raises(ops.KernelError):
        ops.check_status()
    assert ids.tolist() == [[0, 1], [2, 0]] and bool((wt == 0.5).all())
    ops.moe_route_table(torch.tensor([2], dtype=torch.int32).cuda(), table, 8)
    with pytest.raises(ops.KernelError):
        ops.check_status()


def test_heads_normed_without_a_weight_alone():
    """The general preparation with a norm that has no weight, next to the one with weights of one."""
    from jax_vllm_b200 import ops
    g = torch.Generator().manual_seed(9)
    n, Hq, Hk, D, E, P = 11, 4, 2, 24, 8, 8
    proj = torch.randn((n, (Hq + Hk) * D + Hk * E), generator=g).cuda()
    pos, ent = torch.arange(n, dtype=torch.int32).cuda(), torch.zeros(n, dtype=torch.int32).cuda()
    table = torch.tensor([[1, 0]], dtype=torch.int32).cuda()
    freq = tp.banded_frequencies(1e3, 16).float().cuda()
    res = []
    for w, unit_heads in ((torch.ones(D).cuda(), False), (None, True)):
        kc, vc = torch.zeros((2, P, Hk, D)).cuda(), torch.zeros((2, P, Hk, E)).cuda()
        q = torch.empty((n, Hq * D)).cuda()
        ops.head_prepare(proj, 0, Hq * D, (Hq + Hk) * D, q, pos, ent, table, freq, False, w, w, 1e-5, False, None, kc, vc, Hq, Hk,
                         Hk, D, E, unit_heads=unit_heads)
        res.append((q, kc, vc))
    assert all(torch.equal(a, b) for a, b in zip(*res))


# ------------------------------------------------- whole models through the replay class
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_prompt(setup, dtype, tmp_path):
    tag, folder, seqs, want = setup
    steps = whole("r0", seqs["r0"])
    replay(folder, tag, dtype, steps, tmp_path, max_tokens=320)
    compare(steps, tmp_path, CONFIGS[tag]["vocab"], want, dtype, case=f"tidarax {tag}, whole")


@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_last_tokens_one_by_one(setup, dtype, graphs, tmp_path):
    tag, folder, seqs, want = setup
    steps = prefix_then_single("r1", seqs["r1"], tail=25)
    rep = replay(folder, tag, dtype, steps, tmp_path, max_tokens=128, cuda_graphs=graphs)
    compare(steps, tmp_path, CONFIGS[tag]["vocab"], want, dtype, case=f"tidarax {tag}, decoded")
    assert (rep.runner.graph_replays > 0) == graphs


def test_every_token_alone(setup, tmp_path):
    """Token by token from the first one on (no portion at all), in 32-bit, against the prompt run whole."""
    tag, folder, seqs, want = setup
    steps = portions("r3", seqs["r3"], (1,))
    replay(folder, tag, "float32", steps, tmp_path, max_tokens=64)
    compare(steps, tmp_path, CONFIGS[tag]["vocab"], want, "float32", case=f"tidarax {tag}, every token alone")


@pytest.mark.parametrize("sizes", [(2,), (5, 1, 2, 19), (33, 3)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions(setup, dtype, sizes, tmp_path):
    tag, folder, seqs, want = setup
    steps = portions("r2", seqs["r2"], sizes)
    replay(folder, tag, dtype, steps, tmp_path, max_tokens=256)
    compare(steps, tmp_path, CONFIGS[tag]["vocab"], want, dtype, case=f"tidarax {tag}, portions")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_requests_side_by_side_in_reused_pages_and_slots(setup, dtype, tmp_path):
    tag, folder, seqs, want = setup
    seqs = dict(seqs, r0=seqs["r0"][:120])
    steps = mixed_trace(seqs)
    P = PAGE[tag]
    live3 = sum(sorted(-(-len(s) // P) * P for s in seqs.values())[-3:])
    rep = replay(folder, tag, dtype, steps, tmp_path, max_tokens=live3)
    compare(steps, tmp_path, CONFIGS[tag]["vocab"], want, dtype, case=f"tidarax {tag}, side by side")
    assert sum(m["pages_allocated"] for m in rep.records) > rep.cache.num_pages     # pages went out again


def test_schedules_agree_with_each_other_in_32_bit(setup, tmp_path):
    """A position's logits do not depend on the cut, the batch, the pages or the state slot beyond rounding."""
    tag, folder, seqs, _ = setup
    V = CONFIGS[tag]["vocab"]
    seqs = dict(seqs, r0=seqs["r0"][:120])
    a = whole("r0", seqs["r0"])
    b = portions("r0", seqs["r0"], (5, 1, 2, 19))
    c = mixed_trace(seqs)
    replay(folder, tag, "float32", a, tmp_path / "a", 256)
    replay(folder, tag, "float32", b, tmp_path / "b", 256)
    replay(folder, tag, "float32", c, tmp_path / "c", 512)
    ga, gb, gc = (collect(s, tmp_path / d, V)["r0"] for s, d in ((a, "a"), (b, "b"), (c, "c")))
    for pos in ga:
        assert abs(ga[pos] - gb[pos]).max() < 1e-4 and abs(ga[pos] - gc[pos]).max() < 1e-4


def test_trace_run_program(tmp_path):
    """bin/trace_run as a program on a Tidarax folder: stdin steps, `done <step>` lines, files on disk, exit 0."""
    c = CONFIGS["tb"]
    weights = make_weights(c, seed=9)
    folder = write_folder(tmp_path / "model", c, weights)
    seqs = {f"r{i}": random_tokens(n, c["vocab"], seed=40 + i) for i, n in enumerate([40, 21, 33, 12, 18])}
    want = {rid: oracle(c, stored(weights), t) for rid, t in seqs.items()}
    steps = mixed_trace(seqs)
    proc = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32",
                           "--out", str(tmp_path / "out"), "--max-tokens", "192"],
                          input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True,
                          env=dict(os.environ), timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert proc.stdout.split() == [w for s in steps for w in ("done", str(s["step"]))]
    compare(steps, tmp_path / "out", c["vocab"], want, "float32")


# ------------------------------------------------------- weights that make a fault show
def special(tmp_path, c, weights, tokens, dtype, sizes=None, page=16, tail=0):
    from jax_vllm_b200.engine.replay import Replayer
    folder = write_folder(tmp_path / "model", c, weights)
    if tail:
        steps = prefix_then_single("r", tokens, tail=tail)
    else:
        steps = whole("r", tokens) if sizes is None else portions("r", tokens, sizes)
    out = tmp_path / f"out_{dtype}_{sizes}_{tail}"
    rep = Replayer(folder, dtype, out, max_tokens=-(-len(tokens) // 64) * 64, page_size=page)
    rep.run_stream(json.dumps(s) for s in steps)
    return steps, out


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads", ["small", "of_128"])
@pytest.mark.parametrize("far", [0, 1, 15, 16, 63, 64, 255, 256])
def test_one_far_key_among_hundreds(far, heads, dtype, tmp_path):
    """One attention layer in which the last token's query looks for exactly one kind of key: a marker token stands once,
    at a page's, a tile's or a split's edge or at the very start, and only through ANOTHER head's raw score (the score
    matrix is a cyclic shift of heads).  Without it, or without the shift, the plain logits at the last position move by
    far more than the limit; the engine agrees with it whole, in portions and decoding."""
    H, G, D, E = (3, 3, 16, 16) if heads == "small" else (4, 2, 128, 128)
    W, V, n = 64, 40, 330
    c = config(V, W, [layer(H, G, D, E, 4, None, rot=None, scale=0.35 if heads == "small" else 0.06, left=1.0, right=0.01)])
    g = torch.Generator().manual_seed(1)
    weights = make_weights(c, seed=31)
    marker, asker = 7, 9
    emb = weights["embed"]
    emb[:, :8] = 0.0
    emb[marker, :8], emb[asker, :8] = torch.tensor([9.0] + [0.0] * 7), torch.tensor([0.0, 9.0] + [0.0] * 6)
    # the marker's keys and the asker's queries point the same way in every head; other tokens' are small
    direction = torch.randn(D, generator=g)
    for name, heads_n, col in (("q", H, 1), ("k", G, 0)):
        m = 0.02 * torch.randn((heads_n * D, W), generator=g)
        m[:, 8:] *= 1.0
        m[:, col] += direction.repeat(heads_n)
        weights[f"l0.mix.left.{name}"] = m
    T = torch.zeros((H, H))
    for h in range(H):
        T[h, (h + 1) % H] = 1.0
        T[h, h] = -0.2
    weights["l0.mix.left.talk"] = T
    w = stored(weights)
    tokens = [t if t not in (marker, asker) else 11 for t in random_tokens(n, V, seed=77)]
    tokens[far], tokens[-1] = marker, asker
    want = {"r": oracle(c, w, tokens)}
    gone = list(tokens)
    gone[far] = 11
    # the other token's own key and value, and the norm's scale, matter little: the marker's key decides
    assert (oracle(c, w, gone)[-1] - want["r"][-1]).abs().max() > 20 * limits("float32", want["r"])
    straight = dict(w, **{"l0.mix.left.talk": torch.eye(H, dtype=torch.float64)})
    assert (oracle(c, straight, tokens)[-1] - want["r"][-1]).abs().max() > 20 * limits("float32", want["r"])
    for kw in (dict(), dict(sizes=(64, 1, 70)), dict(tail=40)):
        steps, out = special(tmp_path, c, weights, tokens, dtype, **kw)
        compare(steps, out, V, want, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("far", [0, 1, 7, 8, 127, 128, 256])
def test_a_token_far_back_in_the_state(far, dtype, tmp_path):
    """A recurrence that hardly ever lets anything in (a gate bias far below zero) except from one token, 330 tokens long:
    another token at the far position moves the last logits by much more than the limit in the plain implementation, and
    the engine agrees with it whole (runs and tiles of tokens chained), in portions and decoding."""
    V, W = 120, 48
    c = config(V, W, [layer(1, 1, 8, 8, 40, None, left=0.01, right=1.0)])
    weights = make_weights(c, seed=41)
    weights["l0.mix.right.z"] = 0.02 * weights["l0.mix.right.z"]
    weights["l0.mix.right.z.b"] = torch.full((40,), -7.0)
    marker = 5
    weights["embed"][:, 0] = 0.0
    weights["embed"][marker, 0] = 12.0
    weights["l0.mix.right.z"][:, 0] = 3.0                       # the marker opens every gate
    w = stored(weights)
    tokens = [t if t != marker else 6 for t in random_tokens(330, V, seed=78)]
    tokens[far] = marker
    want = {"r": oracle(c, w, tokens)}
    changed = list(tokens)
    changed[far] = 6
    assert (oracle(c, w, changed)[-1] - want["r"][-1]).abs().max() > 20 * limits("float32", want["r"])
    for kw in (dict(), dict(sizes=(64, 1, 70)), dict(sizes=(8, 120)), dict(tail=40)):
        steps, out = special(tmp_path, c, weights, tokens, dtype, **kw)
        compare(steps, out, V, want, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_first_tokens_and_the_added_one(dtype, tmp_path):
    """Scores far below zero: the added one takes nearly all the weight, most of all at the first tokens, where there are
    few keys; dropping it moves the plain logits by far more than the limit at every position."""
    c = config(60, 32, [layer(4, 2, 16, 16, 6, None, scale=0.3, left=2.0, right=0.05),
                        layer(2, 1, 16, 8, 6, dense(24), scale=0.25, left=1.0, right=0.05)])
    weights = make_weights(c, seed=51)
    weights["l0.mix.left.talk"] = -2.5 * torch.eye(4) + 0.2
    w = stored(weights)
    tokens = random_tokens(90, 60, seed=79)
    want = {"r": oracle(c, w, tokens)}
    original = tp.zero_sink_weights
    tp.zero_sink_weights = lambda s, first=0: original(s + 40.0, first)         # the one beside it becomes nothing
    try:
        without = oracle(c, w, tokens)
    finally:
        tp.zero_sink_weights = original
    assert (without - want["r"]).abs().max(dim=1).values.min() > 20 * limits("float32", want["r"])
    for kw in (dict(), dict(sizes=(1, 2, 3)), dict(tail=88)):
        steps, out = special(tmp_path, c, weights, tokens, dtype, **kw)
        compare(steps, out, 60, want, dtype)


def test_long_decoding(tmp_path):
    """600 tokens, the last 450 decoded one by one from captured graphs (over the edges of pages and key splits), in both
    precisions; every tenth position compared."""
    from jax_vllm_b200.engine.replay import Replayer
    c = config(80, 48, [layer(4, 2, 16, 16, 24, moe(4, 2, 16), rot=rotation(16, 1e3, (8.0, 1.0, 4.0, 256)), left=0.9, right=0.8)])
    weights = make_weights(c, seed=61)
    folder = write_folder(tmp_path / "model", c, weights)
    tokens = random_tokens(600, 80, seed=80)
    want = {"r": oracle(c, stored(weights), tokens)}
    steps = prefix_then_single("r", tokens, tail=450)
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        rep = Replayer(folder, dtype, out, max_tokens=640, page_size=16, cuda_graphs=True)
        rep.run_stream(json.dumps(s) for s in steps)
        compare(steps, out, 80, want, dtype)
        assert rep.runner.graph_replays > 400


# ----------------------------------------------------------- generation, scheduler, entry point
def plain_greedy(c, w, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(tp.forward(c, w, seq)[-1].argmax()))
    return seq[len(prompt):]


@pytest.mark.parametrize("tag", ["ta", "te"])
def test_greedy_generation_through_the_entry_point(tag, tmp_path):
    """make_driver + generate: the scheduler's portions, decode steps from captured graphs, sampling; 30 tokens each."""
    from jax_vllm_b200 import SamplingParams, generate, load_from_path, make_driver
    c = CONFIGS[tag]
    weights = make_weights(c, seed=21)
    folder = write_folder(tmp_path / "model", c, weights)
    model = load_from_path(folder, dtype="fp32")
    d = make_driver(model, max_num_seqs=3, max_model_len=96, block_size=16, max_tokens_per_step=16)
    prompts = [random_tokens(n, c["vocab"], seed=50 + n) for n in (21, 5, 40)]
    got = generate(d, prompts, SamplingParams(max_new_tokens=30))
    assert got == [plain_greedy(c, stored(weights), p, 30) for p in prompts]
    assert d.runner.graph_replays > 0
    d.cache.check()


def test_random_arrivals_with_few_pages_and_slots(tmp_path):
    """Requests arrive at random steps into a pool too small for them: the youngest is preempted and run again, pages and
    state slots come back and are used again (a slot's state starts from zero for its next owner); greedy tokens depend
    on none of it."""
    import random
    from jax_vllm_b200 import SamplingParams, add_request, has_work, load_from_path, make_driver, step
    c = CONFIGS["tb"]
    weights = make_weights(c, seed=22)
    folder = write_folder(tmp_path / "model", c, weights)
    rng = random.Random(1)
    model = load_from_path(folder, dtype="fp32")
    d = make_driver(model, max_num_seqs=3, max_model_len=64, block_size=8, num_blocks=9, max_tokens_per_step=24)
    prompts = [random_tokens(rng.randrange(1, 30), c["vocab"], seed=100 + i) for i in range(8)]
    new_tokens = [rng.randrange(6, 27) for _ in prompts]
    waiting, ids = list(range(len(prompts))), {}
    while waiting or has_work(d):
        if waiting and (rng.random() < 0.4 or not has_work(d)):
            i = waiting.pop(0)
            ids[i] = add_request(d, prompts[i], SamplingParams(max_new_tokens=new_tokens[i]))
        step(d)
        d.cache.check()
    assert not d.cache.live
    w = stored(weights)
    for i, prompt in enumerate(prompts):
        assert d.requests[ids[i]].output_ids == plain_greedy(c, w, prompt, new_tokens[i]), f"request {i}"


def test_command_line_and_random_weights(tmp_path):
    """cli.py as a user runs it on a Tidarax folder (the printed ids are the plain implementation's greedy tokens), and on
    a configuration with random weights, whose folder the plain implementation reads."""
    from jax_vllm_b200 import registry
    from jax_vllm_b200.weights.random_init import write_model_folder
    c = CONFIGS["td"]
    weights = make_weights(c, seed=23)
    folders = {"given": write_folder(tmp_path / "model", c, weights),
               "random": write_model_folder(tmp_path / "random", registry.config_from_dict(CONFIGS["ta"]), seed=4)}
    for which, folder in folders.items():
        cfg = tp.read_config(folder)
        w = tp.read_weights(folder)
        prompts = [random_tokens(37, cfg["vocab"], seed=60), random_tokens(37, cfg["vocab"], seed=60)[:33] + [5, 6], [9]]
        cmd = [sys.executable, str(ROOT / "cli.py"), "--model-path", str(folder), "--dtype", "fp32", "--max-tokens", "7",
               "--max-model-len", "128", "--block-size", "32", "--no-prewarm"]
        for p in prompts:
            cmd += ["--prompt-ids", ",".join(map(str, p))]
        proc = subprocess.run(cmd, capture_output=True, text=True, env=dict(os.environ), timeout=600)
        assert proc.returncode == 0, proc.stderr[-2000:]
        got = [json.loads(line)["output_ids"] for line in proc.stdout.splitlines() if line.startswith("{")]
        assert got == [plain_greedy(cfg, w, p, 7) for p in prompts], which


# ------------------------------------------------------------------ configurations drawn at random
def random_configuration(seed):
    import random
    rng = random.Random(seed)
    layers = []
    for _ in range(rng.randrange(1, 5)):
        kv = rng.choice([1, 2, 3, 4])
        dim, vdim = rng.choice([6, 8, 12, 16, 32, 48, 64]), rng.choice([5, 8, 16, 32, 64])
        rot = rng.choice([None, rotation(rng.choice([2, dim // 2 // 2 * 2, dim]), rng.choice([1e3, 1e4, 1e6]),
                                         rng.choice([None, (8.0, 1.0, 4.0, 64), (2.0, 1.0, 2.0, 30)]))])
        mlp = rng.choice([None, dense(rng.choice([8, 24, 40, 130])), moe(rng.choice([1, 3, 6]), 1, rng.choice([8, 16, 30])),
                          moe(5, rng.choice([2, 5]), rng.choice([8, 24]))])
        layers.append(layer(kv * rng.choice([1, 2, 3]), kv, dim, vdim, rng.choice([3, 16, 50, 90]), mlp, rot=rot,
                            scale=rng.choice([None, 0.1, 0.5]), left=rng.choice([0.5, 1.0, 1.7]), right=rng.choice([0.4, 1.0, 1.5])))
    return config(rng.randrange(60, 300), rng.choice([40, 56, 72, 96]), layers, eps=rng.choice([1e-6, 1e-5, 1e-4]))


@pytest.mark.parametrize("seed", range(8))
def test_configurations_drawn_at_random(seed, tmp_path):
    """Layer orders, sizes and constants drawn at random: a prompt whole and in portions, and decoded, in both precisions;
    and five requests side by side in 32-bit."""
    c = random_configuration(seed)
    weights = make_weights(c, seed=60 + seed)
    folder = write_folder(tmp_path / "model", c, weights)
    w = stored(weights)
    page = [4, 8, 16, 32][seed % 4]
    seqs = {f"r{i}": random_tokens(n, c["vocab"], seed=200 + 10 * seed + i) for i, n in enumerate([90, 33, 61, 12, 40])}
    want = {rid: oracle(c, w, t) for rid, t in seqs.items()}
    rounding = {rid: rounding_error(c, w, seqs[rid]) for rid in ("r0", "r2")}
    from jax_vllm_b200.engine.replay import Replayer
    for dtype in ("float32", "bfloat16"):
        for k, steps in enumerate((whole("r0", seqs["r0"]), portions("r0", seqs["r0"], (3, 1, 30, 2)),
                                   prefix_then_single("r2", seqs["r2"], tail=22))):
            out = tmp_path / f"{dtype}_{k}"
            rep = Replayer(folder, dtype, out, max_tokens=128, page_size=page)
            rep.run_stream(json.dumps(s) for s in steps)
            compare(steps, out, c["vocab"], want, dtype, rounding=rounding)
    steps = mixed_trace(seqs)
    rep = Replayer(folder, "float32", tmp_path / "mixed", max_tokens=320, page_size=page)
    rep.run_stream(json.dumps(s) for s in steps)
    rep.cache.check()
    compare(steps, tmp_path / "mixed", c["vocab"], want, "float32")
