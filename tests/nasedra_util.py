"""Test material for the Nasedra design: small configurations that differ in every size and option, and a model-folder
writer that is independent of the product's."""

from __future__ import annotations

import json
from pathlib import Path

import torch


def rotation(dims, base=1e4, scaling=(8.0, 60, 4.0, 0.5)):
    """`scaling` = (factor, original, fast, slow), or None; a small `original` puts pairs at, between and past both ends."""
    r = {"base": base, "dims": dims}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def attention(heads, kv, dim, vdim, rot=None, size=None, keep=0, cap=None, scale=None, kv_from=None):
    mx = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5}
    if rot is not None:
        mx["rot"] = rot
    if size is not None:
        mx["mask"] = {"size": size, "keep_first": keep}
    if cap is not None:
        mx["softcap"] = cap
    if kv_from is not None:
        mx["kv_from"] = kv_from
    return mx


def gla(heads, dim, vdim, tau):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def layer(mixer, mlp):
    return {"type": "gla" if "tau" in mixer else "attention", "mixer": mixer, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, identity=0, scale=1.0, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "scale": scale, "top": top}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def config(vocab, width, layers, eps=1e-5, scale=1.0):
    return {"architecture": "Nasedra", "embedding": {"scale": scale}, "vocab": vocab, "width": width, "layers": layers,
            "norm": {"eps": eps}}


_R8 = rotation(8, 1e3)
# a reader whose window and kept tokens are wider than those of the layer whose keys it reads; a layer without a feed-forward
NA = config(200, 64, [layer(gla(3, 12, 20, 8.0), dense(48)),
                      layer(attention(6, 3, 16, 24, _R8, size=24, keep=3, cap=12.0), moe(5, 2, 24, identity=2, scale=1.7, shared=40)),
                      layer(gla(2, 16, 8, 3.0), moe(4, 1, 16, identity=1, scale=0.8)),
                      layer(attention(6, 3, 16, 24, _R8, size=40, keep=6, cap=9.0, kv_from=1), None)], eps=1e-6, scale=3.0)
# nothing a multiple of 8; no rotation, no cap, no mask in the owner and a window without kept tokens in its reader; every
# expert chosen; the decay's temperature 1
NB = config(131, 72, [layer(attention(4, 1, 10, 7), moe(3, 3, 20, scale=0.9)),
                      layer(gla(1, 7, 9, 1.0), None),
                      layer(attention(4, 1, 10, 7, size=9, cap=5.0, kv_from=0), dense(30)),
                      layer(gla(5, 6, 3, 20.0), moe(6, 3, 22, identity=4, scale=2.0, shared=15))], eps=3e-6, scale=0.7)
# tensor-core sizes: keys and values of two sizes, grouped products of experts on the tensor cores
NC = config(320, 128, [layer(attention(8, 2, 64, 80, rotation(64, 5e5, (4.0, 256, 16.0, 1.0)), size=70, keep=20, cap=30.0),
                             moe(8, 3, 128, identity=3, scale=2.2, shared=128)),
                       layer(gla(2, 64, 128, 12.0), dense(256)),
                       layer(attention(4, 4, 32, 32, rotation(20, 1e4, None), size=33, keep=0), moe(4, 2, 128, identity=1, scale=1.3)),
                       layer(attention(8, 2, 64, 80, rotation(64, 5e5, (4.0, 256, 16.0, 1.0)), cap=25.0, kv_from=0), dense(64))])
# heads of 128: windows within a tile, over several tiles, kept tokens of more than a tile, no window
ND = config(150, 96, [layer(attention(4, 2, 128, 128, rotation(64, 1e4, (2.0, 300, 8.0, 1.0)), size=100, keep=5, cap=15.0), dense(64)),
                      layer(attention(4, 2, 128, 128, rotation(64, 1e4, (2.0, 300, 8.0, 1.0)), size=170, keep=140, kv_from=0), None),
                      layer(attention(3, 1, 128, 128, size=64, keep=1), moe(6, 2, 40, identity=2, scale=1.1, shared=24)),
                      layer(gla(4, 32, 48, 16.0), dense(40)),
                      layer(attention(2, 2, 128, 128, rotation(128, 1e5), cap=20.0), None)], scale=2.0)
# one head, one channel, one expert beside one identity expert, a window of one
NE = config(90, 40, [layer(attention(1, 1, 16, 24, rotation(2, 1e3), size=1, keep=1, cap=3.0), moe(1, 1, 8, identity=1, scale=0.6)),
                     layer(gla(1, 1, 1, 0.5), moe(1, 2, 8, identity=1, shared=3)),
                     layer(attention(1, 1, 16, 24, rotation(2, 1e3), size=3, keep=70, kv_from=0), dense(8))], eps=1e-4, scale=1.5)
CONFIGS = {"na": NA, "nb": NB, "nc": NC, "nd": ND, "ne": NE}
PAGE = {"na": 16, "nb": 8, "nc": 16, "nd": 32, "ne": 4}
RANK = 5            # of the decays' pairs of matrices (only the tensors' shapes say it)


def tensor_shapes(c: dict, rank: int = RANK) -> dict:
    W, V = c["width"], c["vocab"]
    shapes = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    for i, ly in enumerate(c["layers"]):
        p, mx, ml = f"l{i}", ly["mixer"], ly["mlp"]
        H, D, E = mx["heads"], mx["dim"], mx["vdim"]
        shapes[f"{p}.norm1"] = (W,)
        shapes.update({f"{p}.mix.q": (H * D, W), f"{p}.mix.g": (H * E, W), f"{p}.mix.o": (W, H * E)})
        if ly["type"] == "gla":
            shapes.update({f"{p}.mix.k": (H * D, W), f"{p}.mix.v": (H * E, W), f"{p}.mix.norm": (E,), f"{p}.mix.a1": (rank, W),
                           f"{p}.mix.a2": (H * D, rank), f"{p}.mix.a2.b": (H * D,)})
        elif mx.get("kv_from") is None:
            shapes.update({f"{p}.mix.k": (mx["kv_heads"] * D, W), f"{p}.mix.v": (mx["kv_heads"] * E, W)})
        if ml is None:
            continue
        shapes[f"{p}.norm2"] = (W,)
        gated = lambda q, ff: {f"{q}.gate": (ff, W), f"{q}.up": (ff, W), f"{q}.down": (W, ff)}
        if ml["kind"] == "dense":
            shapes.update(gated(f"{p}.mlp", ml["ff"]))
        else:
            n = ml["router"]["experts"] + ml["router"]["identity"]
            shapes.update({f"{p}.mlp.router": (n, W), f"{p}.mlp.correction": (n,)})
            for e in range(ml["router"]["experts"]):
                shapes.update(gated(f"{p}.mlp.e{e}", ml["expert"]["ff"]))
            if "shared" in ml:
                shapes.update(gated(f"{p}.mlp.shared", ml["shared"]["ff"]))
    return shapes


def make_weights(c: dict, seed: int, rank: int = RANK) -> dict:
    """Random float32 weights: matrices N(0, 1.5/sqrt(fan_in)), embedding of order one, norm weights 1 + N(0, 0.1), decay
    biases N(1, 1), corrections N(0, 0.2)."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(c, rank).items():
        z = torch.randn(shape, generator=g, dtype=torch.float32)
        last = name.rsplit(".", 1)[-1]
        if name == "embed":
            out[name] = z
        elif last == "b":
            out[name] = 1.0 + z
        elif last == "correction":
            out[name] = 0.2 * z
        elif len(shape) == 1:
            out[name] = 1.0 + 0.1 * z
        else:
            out[name] = (1.5 / shape[1] ** 0.5) * z
    return out


def stored(weights: dict) -> dict:
    """The values that the folder holds (bfloat16), as float64: both sides compute from the same numbers."""
    return {k: v.to(torch.bfloat16).to(torch.float64) for k, v in weights.items()}


def write_folder(folder, c: dict, weights: dict, dtype=torch.bfloat16) -> Path:
    from safetensors.torch import save_file

    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(c))
    save_file({k: v.to(dtype).contiguous() for k, v in weights.items()}, str(folder / "model.safetensors"))
    return folder
