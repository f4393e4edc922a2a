"""Plain, slow, whole-sequence implementation of the Tidarax design (on the CPU, float64 or float32): the oracle that
the engine is compared with.

No cache, no batching, no kernels: one function per mechanism, token by token where the design is a recurrence.
It shares no code with the product package: it reads config.json keys and safetensors names itself.

The design in this file's notation (x: the stream [tokens, width]; unit(y) = y / sqrt(mean(y^2) + eps)):

    x            = embed[token]
    layer:         x <- x + mixer(unit(x) * (1 + w1));   x <- x + ff(unit(x) * (1 + w2))      (no ff: no second half)
    mixer(u)     = left_scale * left(u) + right_scale * right(u)
        left       q, k rotated (halves, frequencies in three bands), then unit per head; raw score r[g, i, j] =
                   scale * q[i, g] . k[j, g // (H/G)]; s[h] = sum_g T[h, g] r[g]; causal;
                   weight = exp(s) / (1 + sum exp(s)); W_o on the heads side by side
        right      S <- (1 - z) S + z c element by element, z = sigmoid(W_z u + b_z), y = W_x u + b_x, c = y + 1/2 where
                   y >= 0 and sigmoid(y) elsewhere; W_o (S * silu(W_g u))
    ff           dense: W_down act(W_up u), act(z) = a unit(z) + b unit(z^2) + c unit(z^3) + e
                 moe: mean of the experts that the token's id names, expert = W_down (silu(W_gate u) * (W_up u))
    logits       = head (unit(x) * (1 + w))
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
def unit(y: torch.Tensor, eps: float) -> torch.Tensor:
    """y divided by its root mean square over the last axis, eps inside the root."""
    return y / torch.sqrt((y * y).mean(dim=-1, keepdim=True) + eps)


def norm(x, w, eps):
    """RMS norm whose stored weight is around zero."""
    return unit(x, eps) * (1.0 + w)


def silu(z):
    return z * torch.sigmoid(z)


# ---------------------------------------------------------------------------- left
def banded_frequencies(base: float, dims: int, scaling=None) -> torch.Tensor:
    """base^(-2i/dims), i < dims/2, float64.  With scaling {factor, low, high, original}: a wavelength shorter than
    original/high keeps its frequency, one longer than original/low has it divided by the factor, and between the two
    the frequency is a straight mixture of both by where original/wavelength lies between low and high."""
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling is not None:
            factor, low, high = float(scaling["factor"]), float(scaling["low"]), float(scaling["high"])
            original = float(scaling["original"])
            wavelength = 2.0 * math.pi / f
            if wavelength > original / low:
                f = f / factor
            elif not wavelength < original / high:
                s = (original / wavelength - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float64)


def rotate_halves(x, positions, freq):
    """x [T, H, D]: elements i and i + n of every head (n = len(freq)) turn by position * freq[i]; the rest passes."""
    n = len(freq)
    a = positions.to(torch.float64)[:, None] * freq[None, :]
    c, s = torch.cos(a)[:, None, :].to(x.dtype), torch.sin(a)[:, None, :].to(x.dtype)
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], dim=-1)


def raw_scores(q, k, scale):
    """[H, Tq, T]: query head h against key head h // (H / G); q [Tq, H, D], k [T, G, D]."""
    return torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(q.shape[1] // k.shape[1], dim=1)) * scale


def talk(raw, T):
    """The heads' scores mixed: out[h] = sum_g T[h, g] raw[g]."""
    return torch.einsum("hg,gij->hij", T, raw)


def zero_sink_weights(s, first=0):
    """Causal exp(s) / (1 + sum exp(s)) over the keys; s [H, Tq, T], queries at positions first, first + 1, ..."""
    Tq, T = s.shape[1], s.shape[2]
    hidden = torch.arange(T)[None, :] > (first + torch.arange(Tq))[:, None]
    s = s.masked_fill(hidden, -math.inf)
    m = torch.clamp(s.max(dim=-1, keepdim=True).values, min=0.0)
    e = torch.exp(s - m)
    return e / (torch.exp(-m) + e.sum(-1, keepdim=True))


def talking_attend(q, k, v, scale, T, first=0):
    """q [Tq, H, D], k [T, G, D], v [T, G, E] -> [Tq, H, E]."""
    w = zero_sink_weights(talk(raw_scores(q, k, scale), T), first)
    return torch.einsum("hij,jhe->ihe", w, v.repeat_interleave(q.shape[1] // k.shape[1], dim=1))


def attention(u, W, p, mx, eps):
    """u [T, width] -> [T, width]; p the tensor prefix '<layer>.mix.left'."""
    H, G, D, E = int(mx["heads"]), int(mx["kv_heads"]), int(mx["dim"]), int(mx["vdim"])
    n = u.shape[0]
    q = (u @ W[f"{p}.q"].T).view(n, H, D)
    k = (u @ W[f"{p}.k"].T).view(n, G, D)
    v = (u @ W[f"{p}.v"].T).view(n, G, E)
    rot = mx.get("rot")
    if rot is not None:
        freq = banded_frequencies(rot["base"], int(rot["dims"]), rot.get("scaling"))
        pos = torch.arange(n)
        q, k = rotate_halves(q, pos, freq), rotate_halves(k, pos, freq)
    o = talking_attend(unit(q, eps), unit(k, eps), v, float(mx["scale"]), W[f"{p}.talk"])
    return o.reshape(n, H * E) @ W[f"{p}.o"].T


# --------------------------------------------------------------------------- right
def candidate(y):
    return torch.where(y >= 0, y + 0.5, torch.sigmoid(y))


def gru_scan(zl, y, S=None):
    """zl, y [T, C]: the gate's and the candidate's pre-activations, biases included.  Returns (the states after every
    token [T, C], the last one)."""
    z, c = torch.sigmoid(zl), candidate(y)
    S = torch.zeros(zl.shape[1], dtype=zl.dtype) if S is None else S.clone()
    out = torch.zeros_like(zl)
    for t in range(zl.shape[0]):
        S = (1.0 - z[t]) * S + z[t] * c[t]
        out[t] = S
    return out, S


def min_gru(u, W, p):
    """p the tensor prefix '<layer>.mix.right'."""
    S, _ = gru_scan(u @ W[f"{p}.z"].T + W[f"{p}.z.b"], u @ W[f"{p}.x"].T + W[f"{p}.x.b"])
    return (S * silu(u @ W[f"{p}.g"].T)) @ W[f"{p}.o"].T


def parallel_mixer(u, W, p, mx, eps):
    return float(mx["left_scale"]) * attention(u, W, f"{p}.left", mx["left"], eps) + \
        float(mx["right_scale"]) * min_gru(u, W, f"{p}.right")


# -------------------------------------------------------------------- feed-forwards
def poly_norm(z, coef, eps):
    a, b, c, e = coef[0], coef[1], coef[2], coef[3]
    return a * unit(z, eps) + b * unit(z * z, eps) + c * unit(z * z * z, eps) + e


def dense_ff(u, W, p, eps):
    return poly_norm(u @ W[f"{p}.up"].T, W[f"{p}.act"], eps) @ W[f"{p}.down"].T


def expert(u, W, p):
    return (silu(u @ W[f"{p}.gate"].T) * (u @ W[f"{p}.up"].T)) @ W[f"{p}.down"].T


def table_ff(u, W, p, ml, tokens):
    """The experts of a token are the entries of its id's row of the table, each with the weight 1 / top."""
    chosen = W[f"{p}.table"][torch.as_tensor(tokens)].long()
    out = torch.zeros_like(u)
    for e in range(int(ml["router"]["experts"])):
        rows = (chosen == e).any(-1)
        if rows.any():
            out[rows] += expert(u[rows], W, f"{p}.e{e}") / chosen.shape[1]
    return out


# ------------------------------------------------------------------------ the model
def forward(cfg: dict, W: dict, tokens, taps=None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence run whole.  `taps`, a list, receives the stream after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = W["embed"][torch.as_tensor(tokens)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}"
        x = x + parallel_mixer(norm(x, W[f"{p}.norm1"], eps), W, f"{p}.mix", layer["mixer"], eps)
        ml = layer.get("mlp")
        if ml is not None:
            u = norm(x, W[f"{p}.norm2"], eps)
            x = x + (dense_ff(u, W, f"{p}.mlp", eps) if ml["kind"] == "dense" else table_ff(u, W, f"{p}.mlp", ml, tokens))
        if taps is not None:
            taps.append(x.clone())
    return norm(x, W["final.norm"], eps) @ W["head"].T
