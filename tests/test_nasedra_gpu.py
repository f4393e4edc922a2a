"""The Nasedra design in the engine against the plain implementation (tests/plain/nasedra_plain.py): every mechanism
alone, then models of several sizes through the replay program's class (whole, last tokens one by one, portions down
to two tokens, unequal requests side by side in reused pages and state slots), special weights where random ones would
hide a fault, and greedy generation through the entry point and its scheduler."""

from __future__ import annotations

import copy
import json
import math
import os
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from tests.nasedra_util import (CONFIGS, PAGE, attention, config, dense, gla, layer, make_weights, moe, rotation, stored,
                                write_folder)
from tests.plain import nasedra_plain as npl
from tests.test_nufapel_gpu import mixed_trace, scrambled_pages
from tests.test_replay_gpu import limits
from tests.util import collect, portions, prefix_then_single, random_tokens, whole

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
LENGTHS = {"na": [110, 60, 100, 33, 70], "nb": [90, 38, 64, 51, 27], "nc": [200, 90, 150, 40, 66], "nd": [420, 200, 330, 40, 150],
           "ne": [95, 40, 83, 35, 20]}
CLOSE_CALL = 0.05      # a difference of choice scores below which bfloat16 may choose another expert


def oracle(c, w, tokens):
    return npl.forward(c, w, tokens).to(torch.float32)


def rounding_error(c, w, tokens, forced=None):
    """Per position, how far the plain logits move when the operands and the result of every matrix product are
    rounded to bfloat16 and nothing else is: what rounding alone does to this model at this token."""
    bf = lambda x: x.to(torch.bfloat16).to(torch.float64)
    exact = npl.forward(c, w, tokens, forced=forced)
    plain_matmul = torch.Tensor.__matmul__
    torch.Tensor.__matmul__ = lambda a, b: bf(plain_matmul(bf(a), bf(b)))
    try:
        rounded = npl.forward(c, w, tokens, forced=forced)
    finally:
        torch.Tensor.__matmul__ = plain_matmul
    return (rounded - exact).abs().max(dim=1).values


def compare(steps, out_dir, vocab, want, dtype, case=None, rounding=None):
    """Every written row against the oracle's.  32-bit holds every position and the greedy token.  In bfloat16 one
    position in fifty (or one) may be over the limit by up to half of it.  `rounding` (request -> `rounding_error`): a
    bfloat16 position's limit is at least three times what rounding alone does there, and as that is one draw of an
    estimate, one position in ten may then be over."""
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
    assert slightly <= max(1, (0.1 if rounding is not None else 0.02) * total), f"{slightly} of {total} positions are over the limit"
    if case is not None:
        record_worst(case, dtype, worst, lim_of_worst)
    return got


class Routes:
    """Records which experts the engine chose, call by call (a context manager around a replay without captured graphs),
    and puts them back together per request: {request: [one [tokens, top] tensor per routed layer]}."""

    def __enter__(self):
        from jax_vllm_b200 import ops
        self.ops, self.orig, self.calls = ops, ops.moe_route, []

        def recording(*a, **k):
            out = self.orig(*a, **k)
            self.calls.append(out[0].cpu().long())
            return out
        ops.moe_route = recording
        return self

    def __exit__(self, *exc):
        self.ops.moe_route = self.orig
        return False

    def per_request(self, steps, n_routed):
        assert len(self.calls) == n_routed * len(steps)          # every step ran every routed layer once, eagerly
        out = {}
        for k, s in enumerate(steps):
            at = 0
            for e in s["entries"]:
                n = len(e["tokens"])
                for i in range(n_routed):
                    out.setdefault(e["id"], [[] for _ in range(n_routed)])[i].append(self.calls[k * n_routed + i][at:at + n])
                at += n
        return {rid: [torch.cat(parts) for parts in layers] for rid, layers in out.items()}


def run(folder, dtype, steps, out_dir, max_tokens, page, **switches):
    from jax_vllm_b200.engine.replay import Replayer
    rep = Replayer(folder, dtype, out_dir, max_tokens=max_tokens, page_size=page, **switches)
    rep.run_stream(json.dumps(s) for s in steps)
    rep.cache.check()
    assert not rep.cache.live
    return rep


def replay_and_compare(c, w, folder, page, dtype, seqs, want, steps, out_dir, max_tokens, case=None, **switches):
    """The replay against the oracle.  In bfloat16 the plain implementation is made to take the experts that the engine
    took, which may be others than its own only where the choice scores nearly tie."""
    n_routed = sum(1 for ly in c["layers"] if ly["mlp"] is not None and ly["mlp"]["kind"] == "moe")
    if dtype == "float32":
        rep = run(folder, dtype, steps, out_dir, max_tokens, page, **switches)
        compare(steps, out_dir, c["vocab"], want, dtype, case=case)
        return rep
    with Routes() as routes:
        rep = run(folder, dtype, steps, out_dir, max_tokens, page, **switches)
    taken = routes.per_request(steps, n_routed) if n_routed else {e["id"]: [] for s in steps for e in s["entries"]}
    followed, rounding = {}, {}
    for rid, forced in taken.items():
        free = []
        followed[rid] = npl.forward(c, w, seqs[rid], forced=forced, free=free).to(torch.float32)
        for mine, (own, gap) in zip(forced, free):
            differs = (mine.sort(dim=1).values != own.sort(dim=1).values).any(dim=1)
            assert (gap[differs] < CLOSE_CALL).all(), f"{rid}: the engine chose other experts far from a tie"
        rounding[rid] = rounding_error(c, w, seqs[rid], forced=forced)
    compare(steps, out_dir, c["vocab"], followed, dtype, case=case, rounding=rounding)
    return rep


@pytest.fixture(scope="module", params=sorted(CONFIGS))
def setup(request, tmp_path_factory):
    tag = request.param
    c = CONFIGS[tag]
    weights = make_weights(c, seed=5)
    folder = write_folder(tmp_path_factory.mktemp(f"nasedra_{tag}"), c, weights)
    w = stored(weights)
    seqs = {f"r{i}": random_tokens(n, c["vocab"], seed=20 + i) for i, n in enumerate(LENGTHS[tag])}
    want = {rid: oracle(c, w, t) for rid, t in seqs.items()}
    assert all(v.abs().max() > 1.0 for v in want.values())     # logits of order one, not a flat model
    return tag, folder, seqs, want, w


def entries_of(lengths, slots):
    cu = torch.tensor([0] + list(torch.tensor(lengths).cumsum(0)), dtype=torch.int32).cuda()
    return cu, torch.tensor(slots, dtype=torch.int32).cuda()


# ------------------------------------------------------------------ mechanisms alone
KERNELS = {
    # name: (kernel, query heads, key heads, key size, value size, dtype)
    "simt32": ("simt", 6, 3, 20, 12, torch.float32), "simt32_wide": ("simt", 2, 1, 300, 40, torch.float32),
    "simt16": ("simt", 3, 1, 40, 40, torch.bfloat16), "sizes_16": ("general", 4, 2, 32, 64, torch.bfloat16),
    "sizes_64_80": ("general", 8, 1, 64, 80, torch.bfloat16), "sizes_128": ("general", 20, 1, 128, 128, torch.bfloat16),
}


def kept_case(g, ctx_new, P, n_pages, Hq, Hk, D, E, dtype, window, keep):
    """Caches in scrambled pages filled with not-a-number outside the sequences, pages given back that hold nothing visible
    to the entry's first query; (table, k, v, [(keys, values, queries) per entry])."""
    table = scrambled_pages(ctx_new, P, n_pages, g)
    kc = torch.full((n_pages, P, Hk, D), float("nan"), dtype=dtype)
    vc = torch.full((n_pages, P, Hk, E), float("nan"), dtype=dtype)
    parts = []
    for e, (c, q) in enumerate(ctx_new):
        k = (torch.randn((c + q, Hk, D), generator=g) * 1.5).to(dtype)
        v = torch.randn((c + q, Hk, E), generator=g).to(dtype)
        for j in range(c + q):
            page = j // P
            if window and (page + 1) * P <= c - window + 1 and page * P >= keep:
                table[e, page] = -1
            else:
                kc[table[e, page], j % P], vc[table[e, page], j % P] = k[j], v[j]
        parts.append((k.double(), v.double(), (torch.randn((q, Hq, D), generator=g) * 1.5).to(dtype)))
    return table, kc, vc, parts


def check_kept(got, ctx_new, parts, scale, window, keep, cap, tol):
    """Against the plain attention; one more and one fewer visible key changes the plain result by far more than `tol`."""
    at, matters = 0, 0
    for (c, q), (k, v, qs) in zip(ctx_new, parts):
        see = npl.visible(c + q, window, keep, first=c)
        want = npl.attend(qs.double(), k, v, scale, see, cap)
        assert (got[at:at + q] - want).abs().max() < tol * max(1.0, want.abs().max().item()), f"entry at {at}"
        for wrong in ((window + 1, keep), (window - 1, keep), (window, keep + 1), (window, max(keep - 1, 0))):
            if wrong != (window, keep) and wrong[0] > 0:
                other = npl.attend(qs.double(), k, v, scale, npl.visible(c + q, *wrong, first=c), cap)
                matters += int((other - want).abs().max() > 1e-3)
        at += q
    return matters


@pytest.mark.parametrize("window,keep", [(1, 1), (13, 0), (13, 4), (64, 1), (50, 70), (40, 8), (7, 130)])
@pytest.mark.parametrize("name", sorted(KERNELS))
def test_a_window_that_keeps_the_first_tokens_on_the_attention_kernels(name, window, keep):
    """A prompt portion over several tiles behind earlier context, a short prompt from position 0, and single tokens whose
    keys are split into ranges, one of them shorter than the window; capped scores; kept tokens that end within, at and
    past a page, a tile and the window's start."""
    from jax_vllm_b200 import ops
    kernel, Hq, Hk, D, E, dtype = KERNELS[name]
    g = torch.Generator().manual_seed(Hq * D + E + window + 100 * keep)
    P, scale, cap = 8, 1.3 * D ** -0.5, 7.0
    ctx_new = [(137, 45), (0, 3), (230, 1), (5, 1)]
    table, kc, vc, parts = kept_case(g, ctx_new, P, 80, Hq, Hk, D, E, dtype, window, keep)
    n = sum(q for _, q in ctx_new)
    q_all = torch.cat([p[2] for p in parts]).reshape(n, Hq * D).cuda()
    cu, start = torch.tensor([0, 45, 48, 49, 50], dtype=torch.int32).cuda(), torch.tensor([c for c, _ in ctx_new], dtype=torch.int32).cuda()
    out = torch.full((n, Hq * E), float("nan"), dtype=torch.float32).cuda()
    common = (kc.cuda(), vc.cuda(), table.cuda(), cu, start)
    kw = dict(score_cap=cap, keep=keep)
    if kernel == "general":
        assert ops.attn_general_mma_supports(dtype, D, E)
        tpt = ops.attn_general_mma_tokens_per_tile(Hq, Hk)
        go = lambda work, **split: ops.attn_general_mma(q_all, Hq * D, out, *common, work, work.shape[0], Hq, Hk, scale,
                                                        window=window, **kw, **split)
    else:
        tpt = ops.attn_simt_tokens_per_tile(Hq, Hk)
        go = lambda work, **split: ops.attn_simt(q_all, Hq * D, out, *common, work, work.shape[0], Hq, Hk, D, window, scale, **kw, **split)
    tiles = [(0, t) for t in range(0, 45, tpt)] + [(1, t) for t in range(0, 3, tpt)]
    go(torch.tensor(tiles, dtype=torch.int32).cuda())
    go(torch.tensor([(2, 0), (3, 0)], dtype=torch.int32).cuda(), split_size=64, n_splits=max(1, -(-min(231, window + keep) // 64)))
    ops.check_status()
    matters = check_kept(out.cpu().double().view(n, Hq, E), ctx_new, parts, scale, window, keep, cap,
                         2e-5 if dtype == torch.float32 else 2.5e-2)
    assert matters >= 4, "the mask does not matter here"


@pytest.mark.parametrize("cap", [None, 6.0, 60.0])
@pytest.mark.parametrize("window,keep", [(1, 1), (72, 4), (200, 0), (200, 128), (100, 129), (150, 300), (64, 40)])
@pytest.mark.parametrize("Hq,Hk", [(4, 2), (3, 3), (8, 1)])
def test_a_window_that_keeps_the_first_tokens_on_the_tcgen05_prompt_kernel(Hq, Hk, window, keep, cap):
    """Whole 128-row tiles of a prompt portion on heads of 128: context whose pages before the window have been given back
    except those of the kept tokens (which end within, at and past a tile, and past the window's start), a last tile that
    is not full, an entry of one tile from position 0; without a cap, with one that scores exceed, with one far above them."""
    from jax_vllm_b200 import ops
    D, P, scale = 128, 16, 1.3 * 128 ** -0.5
    tpt = ops.attn_tcgen05_tokens_per_tile(Hq, Hk)
    ctx_new = [(300, 2 * tpt + 22), (0, tpt)]
    g = torch.Generator().manual_seed(Hq + window + keep)
    table, kc, vc, parts = kept_case(g, ctx_new, P, 64, Hq, Hk, D, D, torch.bfloat16, window, keep)
    n = sum(q for _, q in ctx_new)
    q_all = torch.cat([p[2] for p in parts]).reshape(n, Hq * D).cuda()
    cu = torch.tensor([0, ctx_new[0][1], n], dtype=torch.int32).cuda()
    start = torch.tensor([c for c, _ in ctx_new], dtype=torch.int32).cuda()
    out = torch.full((n, Hq * D), float("nan"), dtype=torch.bfloat16).cuda()
    tiles = [(e, t) for e, (_, q) in enumerate(ctx_new) for t in range(0, q, tpt)]
    ops.attn_tcgen05(q_all, Hq * D, out, kc.cuda(), vc.cuda(), table.cuda(), cu, start, torch.tensor(tiles, dtype=torch.int32).cuda(),
                     len(tiles), Hq, Hk, D, scale, window=window, keep=keep, score_cap=cap or 0.0)
    ops.check_status()
    check_kept(out.cpu().double().view(n, Hq, D), ctx_new, parts, scale, window, keep, cap, 2.5e-2)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("Hq,Hk,D,E,rot,interleaved", [(6, 3, 16, 8, 8, True), (3, 1, 20, 12, 20, True), (4, 4, 32, 64, 2, False),
                                                       (1, 1, 70, 34, 40, True), (8, 2, 128, 128, 64, True)])
def test_heads_rotated_with_a_gain(Hq, Hk, D, E, rot, interleaved, dtype):
    """YaRN frequencies and the gain of the rotated elements, on queries and keys at far positions in scrambled pages;
    values pass; queries alone give the same queries."""
    from jax_vllm_b200 import ops
    g = torch.Generator().manual_seed(Hq * D + E)
    P, n_pages = 8, 80
    ctx_new = [(37, 21), (0, 3), (480, 1)]
    table = scrambled_pages(ctx_new, P, n_pages, g)
    n = sum(q for _, q in ctx_new)
    pos = torch.cat([torch.arange(c, c + q) for c, q in ctx_new])
    ent = torch.cat([torch.full((q,), e) for e, (_, q) in enumerate(ctx_new)])
    cols = Hq * D + Hk * (D + E)
    proj = (1.5 * torch.randn((n, cols + 3), generator=g)).to(dtype)
    freq, gain = npl.yarn_frequencies(5e4, rot, {"factor": 6.0, "original": 100, "fast": 8.0, "slow": 1.0})
    assert gain > 1.1
    kc, vc = torch.zeros((n_pages, P, Hk, D), dtype=dtype).cuda(), torch.zeros((n_pages, P, Hk, E), dtype=dtype).cuda()
    q_out, q_alone = (torch.empty((n, Hq * D), dtype=dtype).cuda() for _ in range(2))
    args = (pos.int().cuda(), ent.int().cuda(), table.cuda(), freq.float().cuda(), interleaved, None, None, 0.0, False, None)
    ops.head_prepare(proj.cuda(), 3, 3 + Hq * D, 3 + Hq * D + Hk * D, q_out, *args, kc, vc, Hq, Hk, Hk, D, E, gain=gain)
    ops.head_prepare(proj.cuda(), 3, 0, 0, q_alone, *args, None, None, Hq, Hk, Hk, D, E, gain=gain)
    ops.check_status()
    assert torch.equal(q_out, q_alone)
    x = proj.double()

    def turn(t):
        if interleaved:
            return npl.rotate_pairs(t, pos, freq, gain)
        order = [j for i in range(rot // 2) for j in (i, i + rot // 2)] + list(range(rot, D))
        return npl.rotate_pairs(t[..., order], pos, freq, gain)[..., [order.index(d) for d in range(D)]]

    tol = 5e-5 if dtype == torch.float32 else 1.2e-2
    close = lambda a, b: (a.double().cpu() - b).abs().max().item() < tol * max(1.0, b.abs().max().item())
    assert close(q_out.view(n, Hq, D), turn(x[:, 3:3 + Hq * D].view(n, Hq, D)))
    k = turn(x[:, 3 + Hq * D:3 + Hq * D + Hk * D].view(n, Hk, D))
    for t in range(n):
        page, slot = int(table[ent[t], pos[t] // P]), int(pos[t] % P)
        assert close(kc[page, slot], k[t]), t
        assert torch.equal(vc[page, slot].cpu(), proj[t, 3 + Hq * D + Hk * D:3 + cols].view(Hk, E)), t


@pytest.mark.parametrize("first", [[70, 1, 9], [300, 2, 40]])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,D,E,rank,tau", [(3, 12, 20, 5, 8.0), (1, 1, 1, 1, 1.0), (2, 64, 128, 16, 16.0), (5, 7, 9, 40, 0.5),
                                            (1, 200, 33, 3, 2.0), (4, 32, 32, 16, 30.0)])
def test_gated_linear_attention_alone(H, D, E, rank, tau, dtype, first):
    """Decay, scan and gated norm from a given projection: three entries of unequal length in slots given out of order (long
    ones in segments side by side), then a second call that carries on token by token and in short portions; compared with
    the plain mixer run whole on each sequence (identity matrices for its products)."""
    from jax_vllm_b200 import ops
    from jax_vllm_b200.config.model_spec import GatedLinearAttentionSpec
    from jax_vllm_b200.parts import BuildContext
    from jax_vllm_b200.parts.base import StateLayerCache, StepContext
    from jax_vllm_b200.parts.recurrent import GatedLinearAttention
    g = torch.Generator().manual_seed(H * D + E)
    hd, hv = H * D, H * E
    W = 2 * hd + 2 * hv + rank
    eye = torch.eye(W)
    w = {"l.m.q": eye[:hd], "l.m.k": eye[hd:2 * hd], "l.m.v": eye[2 * hd:2 * hd + hv], "l.m.g": eye[2 * hd + hv:2 * hd + 2 * hv],
         "l.m.a1": eye[2 * hd + 2 * hv:], "l.m.a2": torch.randn((hd, rank), generator=g) * rank ** -0.5,
         "l.m.a2.b": 1.0 + torch.randn(hd, generator=g), "l.m.norm": 1.0 + 0.1 * torch.randn(E, generator=g), "l.m.o": torch.eye(hv)}
    w = {k: v.to(torch.bfloat16).float() for k, v in w.items()}
    mx = gla(H, D, E, tau)
    part = GatedLinearAttention(GatedLinearAttentionSpec(W, H, D, E, tau, D ** -0.5, 1e-5, prefix="m"), "l",
                                BuildContext(dtype, torch.device("cuda")))
    part.bind({k: v.to(torch.bfloat16).cuda() for k, v in w.items()})
    second, slots, n_slots = [1, 5, 2], [3, 0, 4], 6
    seqs = [torch.randn((a + b, W), generator=g).to(dtype).float() for a, b in zip(first, second)]
    state = torch.zeros((n_slots,) + part.cache_need().shape, dtype=torch.float32).cuda()
    state[2] = 5.0
    want = [npl.gla(s.double(), {k: v.double() for k, v in w.items()}, "l.m", mx, 1e-5) for s in seqs]
    done = [0] * 3
    for lengths in (first, second):
        rows = torch.cat([seqs[e][done[e]:done[e] + n] for e, n in enumerate(lengths)]).to(dtype).cuda()
        cu, sl = entries_of(lengths, slots)
        step = StepContext(n_tokens=rows.shape[0], n_entries=3, token_ids=None, positions=None, token_entry=None, cu_seqlens=cu,
                           start_pos=None, state_slots=sl, logit_rows=None, n_logit_rows=0, block_tables=[], tile_work={},
                           decode_work=(None, 0), max_seq_len=0)
        out = torch.full((rows.shape[0], hv + 3), 9.0, dtype=dtype).cuda()
        part.from_projection(rows, step, StateLayerCache(state), out[:, 3:])
        ops.check_status()
        assert bool((out[:, :3] == 9.0).all())
        at = 0
        for e, n in enumerate(lengths):
            ref = want[e][done[e]:done[e] + n]
            tol = 5e-5 if dtype == torch.float32 else 3e-2
            assert (out[at:at + n, 3:].double().cpu() - ref).abs().max() < tol * max(1.0, ref.abs().max().item()), (e, lengths)
            at += n
            done[e] += n
    assert bool((state[2] == 5.0).all()) and bool((state[1] == 0.0).all())


@pytest.mark.parametrize("experts,identity,top,scale", [(5, 2, 2, 1.7), (1, 1, 2, 1.0), (40, 9, 6, 2.5), (3, 0, 3, 0.9), (2, 6, 3, 0.5)])
def test_router_with_correction_and_identity_experts(experts, identity, top, scale):
    """Choice by score plus correction (also below zero), weights without it, the identity experts' weights summed; pairs in
    the order of their experts, none for an identity expert."""
    from jax_vllm_b200 import ops
    g = torch.Generator().manual_seed(experts + top)
    n, E = 70, experts + identity
    z = 2.0 * torch.randn((n, E), generator=g)
    correction = torch.randn(E, generator=g) - 1.5
    ids, wt, *own = ops.moe_route(z.cuda(), top, 1, 1, True, "softmax", "max", 1e-20, scale, correction=correction.cuda(), identity=identity)
    want_ids, want_w = npl.route(z.double(), correction.double(), top, scale)
    assert ids.cpu().tolist() == want_ids.tolist() and (wt.cpu() - want_w).abs().max() < 1e-5
    plain = torch.softmax(z.double(), -1).topk(top, dim=-1).indices
    assert top == E or plain.sort(dim=1).values.tolist() != want_ids.sort(dim=1).values.tolist()       # the correction matters
    if identity:
        assert (own[0].cpu() - (want_w * (want_ids >= experts)).sum(-1)).abs().max() < 1e-5
    sorted_token, pos_of, tile_expert, used = ops.moe_align(ids, experts, 8, identity)
    ops.check_status()
    st, po, te = sorted_token.cpu(), pos_of.cpu(), tile_expert.cpu()
    for t in range(n):
        for k in range(top):
            e, p = int(want_ids[t, k]), int(po[t, k])
            assert p == -1 if e >= experts else (int(st[p]) == t and int(te[p // 8]) == e)
    assert int((st >= 0).sum()) == int((want_ids < experts).sum()) and int(used) == int((te >= 0).sum())


@pytest.mark.parametrize("n", [1, 5, 90, 300])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W,F,E,identity,top,shared", [(48, 24, 5, 2, 2, 40), (128, 128, 8, 3, 3, 128), (72, 20, 3, 0, 3, None),
                                                       (66, 15, 2, 4, 3, 9)])
def test_routed_feed_forward_alone(W, F, E, identity, top, shared, dtype, n):
    """Experts, identity experts and the shared expert on both product kernels, as a feed-forward of its own and as the
    part of a joint output product; the plain layer takes the same choice."""
    from jax_vllm_b200 import ops
    from jax_vllm_b200.config.model_spec import RoutedExpertsSpec
    from jax_vllm_b200.parts import BuildContext
    from jax_vllm_b200.parts.routed_experts import RoutedExperts
    ml = moe(E, top, F, identity=identity, scale=1.9, shared=shared)
    w = {k[3:]: v for k, v in make_weights(config(9, W, [layer(gla(1, 1, 1, 1.0), ml)]), 7).items() if k.startswith("l0.mlp")}
    part = RoutedExperts(RoutedExpertsSpec(W, E, top, F, renormalize=True, activation="swiglu", renorm_eps=1e-20, weight_scale=1.9,
                                           correction="correction", identity=identity, shared_size=shared or 0), "",
                         BuildContext(dtype, torch.device("cuda")))
    part.prefix = "mlp"
    if part.shared is not None:
        part.shared.prefix = "mlp.shared"
    part.bind({k: v.to(torch.bfloat16).cuda() for k, v in w.items()})
    x = torch.randn((n, W), generator=torch.Generator().manual_seed(2)).to(dtype)
    with Routes() as routes:
        got = part.forward(x.cuda(), None).tensor().double().cpu()
        ops.check_status()
    want = npl.moe(x.double(), stored(w), "mlp", ml, forced=routes.calls[0])
    tol = 3e-5 if dtype == torch.float32 else 3e-2
    assert (got - want).abs().max() < tol * max(1.0, want.abs().max().item())
    # the part of a joint product: the shared activation beside other columns, the rest handed back
    acts = torch.zeros((n, 8 + part.inner_size), dtype=dtype).cuda()
    rest = part.inner(x.cuda(), None, acts[:, 8:])
    total = rest.tensor().double().cpu()
    if shared is not None:
        total = total + acts[:, 8:].double().cpu() @ stored(w)["mlp.shared.down"].T
    else:
        assert part.out_weight() is None
    assert (total - want).abs().max() < tol * max(1.0, want.abs().max().item())
    assert bool((acts[:, :8] == 0).all())


@pytest.mark.parametrize("form", ["tensor", "parts", "none"])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,hidden,top", [(5, 40, 1), (7, 33, 3), (200, 2048, 4), (3, 8192, 9), (2, 12100, 2)])
def test_two_norms_of_one_sum(n, hidden, top, dtype, form):
    """Two weights on one normed row, after adding a branch's tensor (or the parts of a sum) and routed rows with identity
    experts' own: against the steps apart; for chosen rows the stream stays as it is."""
    from jax_vllm_b200 import ops
    g = torch.Generator().manual_seed(n + hidden)
    h = torch.randn((n, hidden), generator=g)
    rows = torch.randn((2 * n + 3, hidden), generator=g).to(dtype)
    pick = torch.randint(-1, 2 * n + 3, (n, top), generator=g, dtype=torch.int32)
    coef, own = torch.randn((n, top), generator=g), torch.randn((n, hidden), generator=g).to(dtype)
    own_coef = torch.randn(n, generator=g)
    own_coef[0] = 0.0
    w1, w2 = ((1.0 + 0.1 * torch.randn(hidden, generator=g)).to(dtype) for _ in range(2))
    parts = torch.randn((3, n, hidden), generator=g)
    full = h.double() + torch.einsum("ns,nsc->nc", (coef * (pick >= 0)).double(), rows.double()[pick.clamp(min=0).long()])
    full = full + own_coef.double()[:, None] * own.double()
    picked = ops.PickedRows(rows.cuda(), pick.cuda(), coef.cuda(), own.cuda(), own_coef.cuda())
    delta = picked
    if form == "tensor":
        delta = ops.BranchSum(parts[0].to(dtype).cuda(), picked)
        full = full + parts[0].to(dtype).double()
    elif form == "parts":
        delta = ops.BranchSum(ops.PartialSum(parts.cuda()), picked)
        full = full + parts.double().sum(0)
    want1, want2 = npl.norm(full, w1.double(), 1e-5), npl.norm(full, w2.double(), 1e-5)
    tol = 3e-5 if dtype == torch.float32 else 2e-2
    hc = h.cuda()
    some = torch.tensor([n - 1, 0, n // 2], dtype=torch.int32)
    y = ops.rmsnorm(hc, w1.cuda(), 1e-5, dtype, delta=delta, rows=some.cuda())
    assert torch.equal(hc.cpu(), h) and (y.double().cpu() - want1[some.long()]).abs().max() < tol * want1.abs().max()
    assert (delta.tensor().double().cpu() - (full - h.double())).abs().max() < 1e-4 * full.abs().max()
    y1, y2 = ops.rmsnorm(hc, w1.cuda(), 1e-5, dtype, delta=delta, weight2=w2.cuda())
    ops.check_status()
    assert (y1.double().cpu() - want1).abs().max() < tol * want1.abs().max()
    assert (y2.double().cpu() - want2).abs().max() < tol * want2.abs().max()
    assert (hc.double().cpu() - full).abs().max() < 1e-5 * full.abs().max()
    # nothing to add, and a plain tensor
    z1, z2 = ops.rmsnorm(hc, w1.cuda(), 1e-5, dtype, weight2=w2.cuda())
    assert torch.allclose(z1.float(), y1.float(), rtol=1e-2, atol=1e-3) and torch.allclose(z2.float(), y2.float(), rtol=1e-2, atol=1e-3)
    y1, y2 = ops.rmsnorm(hc, w1.cuda(), 1e-5, dtype, delta=parts[1].cuda(), weight2=w2.cuda())
    full = full + parts[1].double()
    assert (y2.double().cpu() - npl.norm(full, w2.double(), 1e-5)).abs().max() < tol * want2.abs().max() * 2


def test_a_row_that_is_not_there_is_reported():
    from jax_vllm_b200 import ops
    rows, w = torch.randn((4, 16)).cuda(), torch.ones(16).cuda()
    for pick, own in (([[4]], True), ([[-2]], True), ([[-1]], False)):
        picked = ops.PickedRows(rows, torch.tensor(pick, dtype=torch.int32).cuda(), torch.ones((1, 1)).cuda(),
                                *((torch.randn((1, 16)).cuda(), torch.ones(1).cuda()) if own else ()))
        ops.rmsnorm(torch.randn((1, 16)).cuda(), w, 1e-5, torch.float32, delta=picked)
        with pytest.raises(ops.KernelError):
            ops.check_status()
        picked.tensor()
        with pytest.raises(ops.KernelError):
            ops.check_status()
    ids = torch.tensor([[0, 7]], dtype=torch.int32).cuda()
    ops.moe_align(ids, 4, 8, identity=4)
    ops.check_status()
    ops.moe_align(ids, 4, 8, identity=3)
    with pytest.raises(ops.KernelError):
        ops.check_status()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_scaled_embedding_and_activation_into_columns(dtype):
    from jax_vllm_b200 import ops
    g = torch.Generator().manual_seed(3)
    table, ids = torch.randn((30, 50), generator=g).to(dtype), torch.tensor([4, 29, 0, 4], dtype=torch.int32)
    out = ops.embed_gather(table.cuda(), ids.cuda(), scale=2.5)
    assert torch.equal(out.cpu(), 2.5 * table.float()[ids.long()])
    ops.embed_gather(table.cuda(), ids.cuda(), out=out, accumulate=True, scale=0.5)
    assert (out.cpu() - 3.0 * table.float()[ids.long()]).abs().max() < 1e-5
    for inter, off in ((24, 8), (30, 3), (128, 16)):
        gu = torch.randn((9, 2 * inter), generator=g).to(dtype)
        wide = torch.full((9, off + inter + 5), 7.0, dtype=dtype).cuda()
        ops.swiglu(gu.cuda(), out=wide[:, off:off + inter])
        want = npl.silu(gu.double()[:, :inter]) * gu.double()[:, inter:]
        assert (wide[:, off:off + inter].double().cpu() - want).abs().max() < (1e-5 if dtype == torch.float32 else 3e-2) * want.abs().max()
        assert bool((wide[:, :off] == 7.0).all() and (wide[:, off + inter:] == 7.0).all())


# ------------------------------------------------- whole models through the replay class
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_prompt(setup, dtype, tmp_path):
    tag, folder, seqs, want, w = setup
    replay_and_compare(CONFIGS[tag], w, folder, PAGE[tag], dtype, seqs, want, whole("r0", seqs["r0"]), tmp_path, 448,
                       case=f"nasedra {tag}, whole")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_last_tokens_one_by_one(setup, dtype, tmp_path):
    tag, folder, seqs, want, w = setup
    steps = prefix_then_single("r1", seqs["r1"], tail=30)
    replay_and_compare(CONFIGS[tag], w, folder, PAGE[tag], dtype, seqs, want, steps, tmp_path, 256, case=f"nasedra {tag}, decoded")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_captured_steps_give_what_eager_ones_give(setup, dtype, tmp_path):
    tag, folder, seqs, want, w = setup
    steps = prefix_then_single("r1", seqs["r1"], tail=20)
    rows = []
    for graphs in (False, True):
        rep = run(folder, dtype, steps, tmp_path / str(graphs), 256, PAGE[tag], cuda_graphs=graphs)
        assert (rep.runner.graph_replays > 0) == graphs
        rows.append(collect(steps, tmp_path / str(graphs), CONFIGS[tag]["vocab"])["r1"])
    assert all(abs(rows[0][p] - rows[1][p]).max() == 0.0 for p in rows[0])


def test_every_token_alone(setup, tmp_path):
    """Token by token from the first one on (no portion at all), in 32-bit, against the prompt run whole."""
    tag, folder, seqs, want, w = setup
    steps = portions("r3", seqs["r3"], (1,))
    replay_and_compare(CONFIGS[tag], w, folder, PAGE[tag], "float32", seqs, want, steps, tmp_path, 64)


@pytest.mark.parametrize("sizes", [(2,), (5, 1, 2, 19), (33, 3), (128, 65)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions(setup, dtype, sizes, tmp_path):
    tag, folder, seqs, want, w = setup
    steps = portions("r2", seqs["r2"], sizes)
    replay_and_compare(CONFIGS[tag], w, folder, PAGE[tag], dtype, seqs, want, steps, tmp_path, 384, case=f"nasedra {tag}, portions")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_requests_side_by_side_in_reused_pages_and_slots(setup, dtype, tmp_path):
    tag, folder, seqs, want, w = setup
    steps = mixed_trace(seqs)
    P = PAGE[tag]
    live3 = sum(sorted(-(-len(s) // P) * P for s in seqs.values())[-3:])
    rep = replay_and_compare(CONFIGS[tag], w, folder, P, dtype, seqs, want, steps, tmp_path, live3, case=f"nasedra {tag}, side by side")
    assert sum(m["pages_allocated"] for m in rep.records) > rep.cache.num_pages     # pages went out again


def test_schedules_agree_with_each_other_in_32_bit(setup, tmp_path):
    """A position's logits do not depend on the cut, the batch, the pages or the state slot beyond rounding."""
    tag, folder, seqs, _, _ = setup
    V = CONFIGS[tag]["vocab"]
    plans = {"a": whole("r0", seqs["r0"]), "b": portions("r0", seqs["r0"], (5, 1, 2, 19)), "c": mixed_trace(seqs)}
    got = {}
    for k, steps in plans.items():
        run(folder, "float32", steps, tmp_path / k, 1152, PAGE[tag])
        got[k] = collect(steps, tmp_path / k, V)["r0"]
    for pos in got["a"]:
        assert abs(got["a"][pos] - got["b"][pos]).max() < 1e-4 and abs(got["a"][pos] - got["c"][pos]).max() < 1e-4


def test_trace_run_program(tmp_path):
    """bin/trace_run as a program on a Nasedra folder: stdin steps, `done <step>` lines, files on disk, exit 0."""
    c = CONFIGS["nb"]
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
def special(tmp_path, c, weights, w, tokens, dtype, want, **kw):
    folder = write_folder(tmp_path / "model", c, weights)
    for k, plan in enumerate((whole("r", tokens), portions("r", tokens, kw.get("sizes", (7, 2))), portions("r", tokens, (64, 1, 70)),
                              prefix_then_single("r", tokens, tail=kw.get("tail", 40)))):
        out = tmp_path / f"{dtype}_{k}"
        replay_and_compare(c, w, folder, 16, dtype, {"r": tokens}, {"r": want}, plan, out, -(-len(tokens) // 64) * 64)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads", ["small", "of_128"])
@pytest.mark.parametrize("place", ["first", "last_kept", "behind_kept", "page_border", "just_outside", "just_inside", "own"])
def test_one_far_key_among_hundreds(place, heads, dtype, tmp_path):
    """One attention layer whose last query looks for exactly one kind of key: a marker token stands once.  Where the mask
    shows it, the plain logits move by far more than the limit without it; where it does not, they stay as they are to the
    last bit.  The engine agrees whole, in portions and decoding."""
    H, G, D, E = (3, 3, 16, 16) if heads == "small" else (4, 2, 128, 128)
    W, V, n, size, keep = 64, 40, 331, 150, 5
    far = {"first": 0, "last_kept": keep - 1, "behind_kept": keep, "page_border": 16, "just_outside": n - 1 - size,
           "just_inside": n - size, "own": n - 2}[place]
    seen = place in ("first", "last_kept", "just_inside", "own")
    c = config(V, W, [layer(attention(H, G, D, E, size=size, keep=keep, cap=50.0, scale=0.5 if heads == "small" else 0.06), None)])
    g = torch.Generator().manual_seed(1)
    weights = make_weights(c, seed=31)
    marker, asker = 7, 9
    emb = weights["embed"]
    emb[:, :8] = 0.0
    emb[marker, 0], emb[asker, 1] = 9.0, 9.0
    direction = torch.randn(D, generator=g)
    for name, heads_n, col in (("q", H, 1), ("k", G, 0)):
        m = 0.02 * torch.randn((heads_n * D, W), generator=g)
        m[:, col] += direction.repeat(heads_n)
        weights[f"l0.mix.{name}"] = m
    w = stored(weights)
    tokens = [t if t not in (marker, asker) else 11 for t in random_tokens(n, V, seed=77)]
    tokens[far], tokens[-1] = marker, asker
    want = oracle(c, w, tokens)
    gone = list(tokens)
    gone[far] = 11
    moved = (oracle(c, w, gone)[-1] - want[-1]).abs().max()
    assert moved > 20 * limits("float32", want) if seen else moved == 0.0
    special(tmp_path, c, weights, w, tokens, dtype, want)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim", [16, 128])
def test_every_constant_of_the_attention_shows(dim, dtype, tmp_path):
    """Sharp attention (queries and keys larger): a window or a number of kept tokens that is one off in the owner or in its
    reader, another cap, a rotation without its gain or with plain frequencies, a reader that has its own mask taken for the
    owner's: each moves the plain logits by far more than the limit; the engine agrees with the true ones."""
    rot = rotation(8, 1e3, (8.0, 60, 4.0, 0.5))
    c = config(160, 64, [layer(attention(4, 2, dim, dim, rot, size=24, keep=3, cap=6.0), dense(48)),
                         layer(attention(4, 2, dim, dim, rot, size=61, keep=7, cap=8.0, kv_from=0), None)], scale=1.3)
    weights = make_weights(c, seed=31)
    for name in ("l0.mix.q", "l0.mix.k", "l1.mix.q"):
        weights[name] = 2.0 * weights[name]
    w = stored(weights)
    tokens = random_tokens(170, c["vocab"], seed=77)
    want = oracle(c, w, tokens)
    mix = lambda k, i: k["layers"][i]["mixer"]
    changes = [lambda k, i=i, key=key, d=d: mix(k, i)["mask"].__setitem__(key, mix(k, i)["mask"][key] + d)
               for i in (0, 1) for key in ("size", "keep_first") for d in (1, -1)]
    changes += [lambda k, i=i: mix(k, i).__setitem__("softcap", 60.0) for i in (0, 1)]
    changes += [lambda k: mix(k, 1).__setitem__("mask", dict(mix(k, 0)["mask"])), lambda k: k["embedding"].__setitem__("scale", 1.0)]
    for number, change in enumerate(changes):
        other = copy.deepcopy(c)
        change(other)
        assert (oracle(other, w, tokens) - want).abs().max().item() > 20 * limits("float32", want), number
    exact = npl.yarn_frequencies
    for wrong in (lambda *a: (exact(*a)[0], 1.0), lambda b, d, s=None: (exact(b, d)[0], exact(b, d, s)[1])):
        npl.yarn_frequencies = wrong
        try:
            assert (oracle(c, w, tokens) - want).abs().max().item() > 20 * limits("float32", want)
        finally:
            npl.yarn_frequencies = exact
    special(tmp_path, c, weights, w, tokens, dtype, want, tail=60)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("far", [0, 1, 63, 64, 200])
def test_a_token_far_back_in_the_state(far, dtype, tmp_path):
    """A state that hardly forgets (a decay bias far above zero) and takes much from one kind of token, over 330 tokens:
    another token at one far position moves the last logits by much more than the limit in the plain implementation, and
    the engine agrees with it whole (segments side by side), in portions and decoding."""
    c = config(120, 48, [layer(gla(2, 16, 12, 4.0), None)])
    weights = make_weights(c, seed=41)
    weights["l0.mix.a2.b"] = torch.full((32,), 12.0)
    marker = 5
    weights["embed"][:, 0] = 0.0
    weights["embed"][marker, 0] = 12.0
    for name in ("k", "v"):
        weights[f"l0.mix.{name}"][:, 0] *= 4.0
    w = stored(weights)
    tokens = [t if t != marker else 6 for t in random_tokens(330, c["vocab"], seed=78)]
    tokens[far] = marker
    want = oracle(c, w, tokens)
    changed = list(tokens)
    changed[far] = 6
    assert (oracle(c, w, changed)[-1] - want[-1]).abs().max().item() > 20 * limits("float32", want)
    special(tmp_path, c, weights, w, tokens, dtype, want)


def test_long_decoding(tmp_path):
    """600 tokens, the last 450 decoded one by one from captured graphs (over the edges of pages, windows and key splits),
    in both precisions; a dense model, so that no choice of experts needs following."""
    c = config(80, 48, [layer(gla(2, 16, 16, 6.0), dense(32)),
                        layer(attention(4, 2, 16, 16, rotation(16, 1e3, (8.0, 256, 8.0, 1.0)), size=300, keep=9, cap=10.0), dense(40)),
                        layer(attention(4, 2, 16, 16, rotation(16, 1e3, (8.0, 256, 8.0, 1.0)), size=40, keep=2, kv_from=1), None)])
    weights = make_weights(c, seed=61)
    folder = write_folder(tmp_path / "model", c, weights)
    w = stored(weights)
    tokens = random_tokens(600, 80, seed=80)
    want = {"r": oracle(c, w, tokens)}
    steps = prefix_then_single("r", tokens, tail=450)
    for dtype in ("float32", "bfloat16"):
        rep = run(folder, dtype, steps, tmp_path / dtype, 640, 16, cuda_graphs=True)
        compare(steps, tmp_path / dtype, 80, want, dtype, rounding={"r": rounding_error(c, w, tokens)})
        assert rep.runner.graph_replays > 400
        assert rep.records[-2]["pages_free"][0] > 10             # the pages that the windows have passed came back


# ----------------------------------------------------------- generation, scheduler, entry point
def plain_greedy(c, w, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(npl.forward(c, w, seq)[-1].argmax()))
    return seq[len(prompt):]


@pytest.mark.parametrize("tag", ["na", "nd"])
def test_greedy_generation_through_the_entry_point(tag, tmp_path):
    """make_driver + generate: the scheduler's portions, decode steps from captured graphs, sampling; 30 tokens each
    (decoding passes over the ends of windows)."""
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


def test_prefix_reuse_under_windows_that_keep_the_first_tokens(tmp_path):
    """A model of attention layers only: a second request takes the pages of a known prefix (kept ones and the window's) and
    generates what it would have without them."""
    from jax_vllm_b200 import SamplingParams, generate, load_from_path, make_driver
    rot = rotation(8, 1e3)
    c = config(90, 40, [layer(attention(4, 2, 16, 8, rot, size=20, keep=6, cap=9.0), dense(24)),
                        layer(attention(2, 1, 8, 8, size=11, keep=1), moe(3, 1, 16, identity=1)),
                        layer(attention(4, 2, 16, 8, rot, size=26, keep=3, kv_from=0), None)])
    weights = make_weights(c, seed=24)
    model = load_from_path(write_folder(tmp_path / "model", c, weights), dtype="fp32")
    d = make_driver(model, max_num_seqs=2, max_model_len=96, block_size=8, max_tokens_per_step=16)
    base = random_tokens(60, c["vocab"], seed=70)
    w = stored(weights)
    for prompt in (base, base[:50] + [3, 4, 5], base[:33], base):
        assert generate(d, [prompt], SamplingParams(max_new_tokens=12)) == [plain_greedy(c, w, prompt, 12)]
        d.cache.check()
    assert d.cache.stats["prefix_hit_tokens"] >= 48 + 32 + 56


def test_random_arrivals_with_few_pages_and_slots(tmp_path):
    """Requests arrive at random steps into a pool too small for them: the youngest is preempted and run again, pages and
    state slots come back and are used again (a slot's state starts from zero for its next owner); greedy tokens depend
    on none of it."""
    import random
    from jax_vllm_b200 import SamplingParams, add_request, has_work, load_from_path, make_driver, step
    c = CONFIGS["nb"]
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
    """cli.py as a user runs it on a Nasedra folder (the printed ids are the plain implementation's greedy tokens), and on
    a configuration with random weights, whose folder the plain implementation reads."""
    from jax_vllm_b200 import registry
    from jax_vllm_b200.weights.random_init import write_model_folder
    c = CONFIGS["ne"]
    weights = make_weights(c, seed=23)
    folders = {"given": write_folder(tmp_path / "model", c, weights),
               "random": write_model_folder(tmp_path / "random", registry.config_from_dict(CONFIGS["na"]), seed=4)}
    for which, folder in folders.items():
        cfg = npl.read_config(folder)
        w = npl.read_weights(folder)
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
    layers, owners = [], []
    for i in range(rng.randrange(2, 6)):
        if rng.random() < 0.45:
            mixer = gla(rng.choice([1, 2, 3]), rng.choice([3, 8, 16, 30]), rng.choice([4, 8, 17, 32]), rng.choice([0.7, 4.0, 16.0]))
        else:
            mask = rng.choice([{}, dict(size=rng.randrange(1, 70), keep=rng.choice([0, 1, 4, 30]))])
            cap = rng.choice([None, 3.0, 15.0])
            if owners and rng.random() < 0.5:
                j = rng.choice(owners)
                own = layers[j]["mixer"]
                mixer = attention(own["heads"], own["kv_heads"], own["dim"], own["vdim"], own.get("rot"), cap=cap, kv_from=j, **mask)
            else:
                kv, dim = rng.choice([1, 2, 3, 4]), rng.choice([6, 8, 16, 32, 48, 64, 128])
                rot = rng.choice([None, rotation(rng.choice([2, dim // 2 // 2 * 2, dim]), rng.choice([1e3, 1e4, 1e6]),
                                                 rng.choice([None, (8.0, 64, 8.0, 0.5), (2.0, 30, 2.0, 1.0)]))])
                mixer = attention(kv * rng.choice([1, 2, 3]), kv, dim, rng.choice([5, 8, 16, 32, 64, 128]), rot, cap=cap,
                                  scale=rng.choice([None, 0.1, 0.3]), **mask)
                owners.append(i)
        mlp = rng.choice([None, dense(rng.choice([8, 24, 30, 130])),
                          moe(rng.choice([1, 3, 6]), 1, rng.choice([8, 16, 30]), identity=rng.choice([0, 1, 3]), scale=1.5),
                          moe(5, rng.choice([2, 5]), rng.choice([8, 24]), identity=2, scale=rng.choice([0.5, 2.0]), shared=rng.choice([9, 16]))])
        layers.append(layer(mixer, mlp))
    return config(rng.randrange(60, 300), rng.choice([40, 56, 70, 96]), layers, eps=rng.choice([1e-6, 1e-5, 1e-4]),
                  scale=rng.choice([0.5, 1.0, 8.0]))


@pytest.mark.parametrize("seed", range(10))
def test_configurations_drawn_at_random(seed, tmp_path):
    """Layer orders, sizes and constants drawn at random: a prompt whole and in portions, and decoded, in both precisions;
    and five requests side by side in 32-bit."""
    c = random_configuration(seed)
    weights = make_weights(c, seed=60 + seed, rank=[1, 4, 16, 7][seed % 4])
    folder = write_folder(tmp_path / "model", c, weights)
    w = stored(weights)
    page = [4, 8, 16, 32][seed % 4]
    seqs = {f"r{i}": random_tokens(n, c["vocab"], seed=200 + 10 * seed + i) for i, n in enumerate([90, 33, 61, 12, 40])}
    want = {rid: oracle(c, w, t) for rid, t in seqs.items()}
    for dtype in ("float32", "bfloat16"):
        for k, steps in enumerate((whole("r0", seqs["r0"]), portions("r0", seqs["r0"], (3, 1, 30, 2)),
                                   prefix_then_single("r2", seqs["r2"], tail=22))):
            replay_and_compare(c, w, folder, page, dtype, seqs, want, steps, tmp_path / f"{dtype}_{k}", 128)
    replay_and_compare(c, w, folder, page, "float32", seqs, want, mixed_trace(seqs), tmp_path / "mixed", 320)
