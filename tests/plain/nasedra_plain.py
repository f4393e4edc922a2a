"""Plain, slow, whole-sequence implementation of the Nasedra design (on the CPU, float64 or float32): the oracle that
the engine is compared with.

No cache, no batching, no kernels: one function per mechanism, token by token where the design is a recurrence.
It shares no code with the product package: it reads config.json keys and safetensors names itself.

The design in this file's notation (x: the stream [tokens, width]; norm(x, w) = x / sqrt(mean(x^2) + eps) * w):

    x            = embed[token] * embedding.scale
    layer:         x <- x + mixer(norm(x, w1)) + ff(norm(x, w2))          both of the same x; a layer may have no ff
    attention      q, k rotated (pairs 2i, 2i+1; YaRN frequencies, cos and sin times a gain); s = cap tanh(q.k scale / cap);
                   key j of query i: j <= i and (i - j < size or j < keep_first); softmax; heads * sigmoid(W_g u); W_o.
                   With kv_from = j the rotated keys and the values are those of layer j.
    gla            S <- diag(a) S + k v^T, o = S^T q / sqrt(dim), a = sigmoid(W_a2 W_a1 u + b)^(1/tau) per key channel;
                   W_o (norm(o, w) per head * silu(W_g u))
    ff             dense: W_down (silu(W_gate u) * (W_up u))
                   moe: r = softmax(W_router u) over experts + identity; the `top` largest of r + correction; weights
                   r / (their sum + 1e-20) * scale; the last `identity` ones give u itself; plus a shared expert
    logits       = head norm(x, w)
"""

from __future__ import annotations

import json
import math
from pathlib import Path

import torch


def read_config(folder) -> dict:
    return json.loads((Path(folder) / "config.json").read_text())


def read_weights(folder, dtype=torch.float64) -> dict:
    from safetensors import safe_open

    out = {}
    for shard in sorted(Path(folder).glob("*.safetensors")):
        with safe_open(str(shard), framework="pt") as f:
            for key in f.keys():
                t = f.get_tensor(key)
                out[key] = t.to(dtype) if t.is_floating_point() else t
    return out


# ----------------------------------------------------------------------- small parts
def norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def embed(tokens, table, scale):
    return table[torch.as_tensor(tokens)] * scale


# ------------------------------------------------------------------------- attention
def yarn_frequencies(base: float, dims: int, scaling=None):
    """(base^(-2i/dims), i < dims/2, as float64; the gain of cos and sin).  With scaling {factor, original, fast, slow}:
    pairs that turn more than `fast` times over `original` positions keep their frequency, pairs that turn fewer than
    `slow` times have it divided by the factor, and between the two pair numbers the share of the divided one grows
    linearly; the gain is 1 + ln(factor) / 10."""
    freq = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return torch.tensor(freq, dtype=torch.float64), 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def pair_that_turns(times):
        return dims * math.log(original / (2.0 * math.pi * times)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_that_turns(float(scaling["fast"]))), 0)
    hi = min(math.ceil(pair_that_turns(float(scaling["slow"]))), dims - 1)
    for i, f in enumerate(freq):
        share = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        freq[i] = f / factor * share + f * (1.0 - share)
    return torch.tensor(freq, dtype=torch.float64), 0.1 * math.log(factor) + 1.0


def rotate_pairs(x, positions, freq, gain=1.0):
    """x [T, H, D]: elements 2i and 2i + 1 of every head (i < len(freq)) turn by position * freq[i] and grow by `gain`;
    the rest passes."""
    n = 2 * len(freq)
    a = positions.to(torch.float64)[:, None] * freq[None, :]
    c, s = (gain * torch.cos(a))[:, None, :].to(x.dtype), (gain * torch.sin(a))[:, None, :].to(x.dtype)
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    turned = torch.stack([u * c - v * s, v * c + u * s], dim=-1).flatten(-2)
    return torch.cat([turned, x[..., n:]], dim=-1)


def visible(T, window=None, keep_first=0, first=0, rows=None):
    """[rows, T] booleans: which keys the queries at positions first, first + 1, ... see."""
    i = first + torch.arange(T - first if rows is None else rows)[:, None]
    j = torch.arange(T)[None, :]
    see = j <= i
    if window is not None:
        see = see & ((i - j < window) | (j < keep_first))
    return see


def capped(s, cap=None):
    return s if cap is None else cap * torch.tanh(s / cap)


def attend(q, k, v, scale, see, cap=None):
    """q [Tq, H, D], k [T, G, D], v [T, G, E], see [Tq, T] -> [Tq, H, E]."""
    r = q.shape[1] // k.shape[1]
    s = capped(torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(r, dim=1)) * scale, cap)
    w = torch.softmax(s.masked_fill(~see, -math.inf), dim=-1)
    return torch.einsum("hij,jhe->ihe", w, v.repeat_interleave(r, dim=1))


def attention(u, W, p, mx, kept):
    """u [T, width] -> ([T, width], (rotated keys, values)); `kept`: the keys and values of the layer that the mixer's
    `kv_from` names, or None."""
    H, G, D, E = int(mx["heads"]), int(mx["kv_heads"]), int(mx["dim"]), int(mx["vdim"])
    n = u.shape[0]
    pos = torch.arange(n)
    rot = mx.get("rot")
    turn = lambda t: t
    if rot is not None:
        freq, gain = yarn_frequencies(rot["base"], int(rot["dims"]), rot.get("scaling"))
        turn = lambda t: rotate_pairs(t, pos, freq, gain)
    q = turn((u @ W[f"{p}.q"].T).view(n, H, D))
    if kept is None:
        kept = (turn((u @ W[f"{p}.k"].T).view(n, G, D)), (u @ W[f"{p}.v"].T).view(n, G, E))
    mask = mx.get("mask") or {}
    see = visible(n, mask.get("size"), int(mask.get("keep_first", 0)))
    cap = mx.get("softcap")
    o = attend(q, *kept, float(mx["scale"]), see, None if cap is None else float(cap)).reshape(n, H * E)
    return (o * torch.sigmoid(u @ W[f"{p}.g"].T)) @ W[f"{p}.o"].T, kept


# ------------------------------------------------------------- gated linear attention
def channel_decay(z, tau):
    """sigmoid(z)^(1/tau)."""
    return torch.exp(torch.nn.functional.logsigmoid(z) / tau)


def gla_scan(q, k, v, a, S=None):
    """q, k, a [T, H, D], v [T, H, E]; S [H, D, E].  Returns (o [T, H, E], the last S)."""
    T, H, D = k.shape
    S = torch.zeros((H, D, v.shape[2]), dtype=k.dtype) if S is None else S.clone()
    out = torch.zeros((T, H, v.shape[2]), dtype=k.dtype)
    for t in range(T):
        S = a[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(dim=1)
    return out, S


def gla(u, W, p, mx, eps):
    H, D, E, n = int(mx["heads"]), int(mx["dim"]), int(mx["vdim"]), u.shape[0]
    q = (u @ W[f"{p}.q"].T).view(n, H, D) * D ** -0.5
    k = (u @ W[f"{p}.k"].T).view(n, H, D)
    v = (u @ W[f"{p}.v"].T).view(n, H, E)
    z = (u @ W[f"{p}.a1"].T) @ W[f"{p}.a2"].T + W[f"{p}.a2.b"]
    o, _ = gla_scan(q, k, v, channel_decay(z, float(mx["tau"])).view(n, H, D))
    o = norm(o, W[f"{p}.norm"], eps).reshape(n, H * E)
    return (o * silu(u @ W[f"{p}.g"].T)) @ W[f"{p}.o"].T


# -------------------------------------------------------------------- feed-forwards
def gated(u, W, p):
    return (silu(u @ W[f"{p}.gate"].T) * (u @ W[f"{p}.up"].T)) @ W[f"{p}.down"].T


def route(z, correction, top, scale):
    """(chosen [T, top], their weights) from the router's logits [T, experts + identity]."""
    s = torch.softmax(z, dim=-1)
    chosen = (s + correction).topk(top, dim=-1).indices
    w = torch.gather(s, 1, chosen)
    return chosen, w / (w.sum(-1, keepdim=True) + 1e-20) * scale


def moe(u, W, p, ml, forced=None, free=None):
    """`forced` [T, top], if given, replaces the router's choice (the weights still come from the scores); `free`, a list,
    receives (the router's own choice, how far its last chosen score lies above the best one left out)."""
    ro = ml["router"]
    E, top, scale = int(ro["experts"]), int(ro["top"]), float(ro["scale"])
    z = u @ W[f"{p}.router"].T
    ids, w = route(z, W[f"{p}.correction"], top, scale)
    if free is not None:
        order = (torch.softmax(z, dim=-1) + W[f"{p}.correction"]).sort(dim=-1, descending=True).values
        gap = order[:, top - 1] - order[:, top] if top < order.shape[1] else torch.full_like(order[:, 0], math.inf)
        free.append((ids, gap))
    if forced is not None:
        s = torch.gather(torch.softmax(z, dim=-1), 1, forced)
        ids, w = forced, s / (s.sum(-1, keepdim=True) + 1e-20) * scale
    out = torch.zeros_like(u)
    for e in range(E + int(ro.get("identity", 0))):
        weight = (w * (ids == e)).sum(-1, keepdim=True)
        rows = (ids == e).any(-1)
        if rows.any():
            out[rows] += weight[rows] * (gated(u[rows], W, f"{p}.e{e}") if e < E else u[rows])
    if ml.get("shared") is not None:
        out = out + gated(u, W, f"{p}.shared")
    return out


# ------------------------------------------------------------------------ the model
def forward(cfg: dict, W: dict, tokens, taps=None, forced=None, free=None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence run whole.  `taps`, a list, receives the stream after every layer; `forced` (one
    tensor a routed layer) and `free` as for `moe`."""
    eps = float(cfg["norm"]["eps"])
    x = embed(tokens, W["embed"], float(cfg["embedding"]["scale"]))
    kept, forced = {}, list(forced or [])
    for i, layer in enumerate(cfg["layers"]):
        p, mx, ml = f"l{i}", layer["mixer"], layer.get("mlp")
        u = norm(x, W[f"{p}.norm1"], eps)
        if layer["type"] == "attention":
            y, kept[i] = attention(u, W, f"{p}.mix", mx, kept[mx["kv_from"]] if mx.get("kv_from") is not None else None)
        else:
            y = gla(u, W, f"{p}.mix", mx, eps)
        if ml is not None:
            u = norm(x, W[f"{p}.norm2"], eps)
            if ml["kind"] == "dense":
                y = y + gated(u, W, f"{p}.mlp")
            else:
                y = y + moe(u, W, f"{p}.mlp", ml, forced.pop(0) if forced else None, free)
        x = x + y
        if taps is not None:
            taps.append(x.clone())
    return norm(x, W["final.norm"], eps) @ W["head"].T
