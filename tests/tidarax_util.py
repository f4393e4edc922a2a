"""Test material for the Tidarax design: small configurations that differ in every size and option, and a model-folder
writer that is independent of the product's."""

from __future__ import annotations

import json
from pathlib import Path

import torch


def rotation(dims, base=1e4, scaling=(4.0, 1.0, 4.0, 64)):
    """`scaling` = (factor, low, high, original): a small `original` puts frequencies into all three bands."""
    r = {"base": base, "dims": dims}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return r


def layer(heads, kv, dim, vdim, gru, mlp, rot="whole", scale=None, left=1.0, right=1.0):
    """A layer of attention (left) beside a recurrence (right); `rot`: "whole", None, or the rotation's dictionary."""
    le = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5}
    if rot is not None:
        le["rot"] = rotation(dim) if rot == "whole" else rot
    return {"type": "parallel", "mixer": {"left": le, "right": {"width": gru}, "left_scale": left, "right_scale": right},
            "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(vocab, width, layers, eps=1e-5):
    return {"architecture": "Tidarax", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}}


# three key heads under six query heads, values narrower than keys, rotation over part of a head, layers of other sizes
# and scales, several experts a token
TA = config(200, 64, [layer(6, 3, 16, 8, 40, dense(48), rot=rotation(8, 1e3), left=0.7, right=1.3),
                      layer(4, 1, 32, 48, 72, moe(5, 3, 24), left=1.5, right=0.6),
                      layer(2, 2, 24, 16, 16, moe(3, 1, 16), rot=rotation(24, 5e4, None), left=-0.9, right=0.8)], eps=1e-6)
# nothing a multiple of 8, no rotation in a layer, a layer without a feed-forward, all experts for every token
TB = config(131, 72, [layer(3, 3, 10, 7, 33, None, rot=rotation(6, 1e4, (8.0, 1.0, 4.0, 40)), left=1.1, right=0.9),
                      layer(5, 1, 21, 12, 50, moe(4, 4, 20), rot=None, left=0.5, right=2.0),
                      layer(2, 1, 20, 20, 9, dense(100), left=1.0, right=1.0)], eps=3e-6)
# tensor-core sizes: key rows of 256 and 128, grouped products of experts on the tensor cores, widths over 128
TC = config(320, 128, [layer(8, 4, 64, 64, 256, moe(8, 2, 128), left=0.8, right=1.1),
                       layer(4, 2, 64, 32, 128, dense(256), scale=0.2, left=1.2, right=0.7),
                       layer(4, 4, 96, 32, 64, dense(64), left=0.9, right=1.0)], eps=1e-5)
# one layer, one head, one channel
TD = config(90, 40, [layer(1, 1, 16, 24, 1, dense(8), left=0.6, right=1.4)], eps=1e-4)
# heads of 128 with values of 128: two, four and eight key heads, one of them under a single query head each
TE = config(150, 96, [layer(4, 2, 128, 128, 48, dense(64), rot=rotation(64, 1e4, (8.0, 1.0, 4.0, 256)), left=0.75, right=1.25),
                      layer(8, 4, 128, 128, 32, moe(6, 2, 40), left=1.1, right=0.85),
                      layer(8, 8, 128, 128, 20, None, rot=rotation(128, 1e5, (2.0, 1.0, 8.0, 100)), left=0.9, right=0.95)],
            eps=1e-5)
CONFIGS = {"ta": TA, "tb": TB, "tc": TC, "td": TD, "te": TE}
PAGE = {"ta": 16, "tb": 8, "tc": 16, "td": 4, "te": 32}


def tensor_shapes(c: dict) -> dict:
    W, V = c["width"], c["vocab"]
    shapes = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    for i, ly in enumerate(c["layers"]):
        p, le, ri, ml = f"l{i}", ly["mixer"]["left"], ly["mixer"]["right"], ly["mlp"]
        H, G, D, E, C = le["heads"], le["kv_heads"], le["dim"], le["vdim"], ri["width"]
        shapes[f"{p}.norm1"] = (W,)
        shapes.update({f"{p}.mix.left.q": (H * D, W), f"{p}.mix.left.k": (G * D, W), f"{p}.mix.left.v": (G * E, W),
                       f"{p}.mix.left.talk": (H, H), f"{p}.mix.left.o": (W, H * E), f"{p}.mix.right.z": (C, W),
                       f"{p}.mix.right.z.b": (C,), f"{p}.mix.right.x": (C, W), f"{p}.mix.right.x.b": (C,),
                       f"{p}.mix.right.g": (C, W), f"{p}.mix.right.o": (W, C)})
        if ml is None:
            continue
        shapes[f"{p}.norm2"] = (W,)
        if ml["kind"] == "dense":
            shapes.update({f"{p}.mlp.up": (ml["ff"], W), f"{p}.mlp.down": (W, ml["ff"]), f"{p}.mlp.act": (4,)})
        else:
            F = ml["expert"]["ff"]
            shapes[f"{p}.mlp.table"] = (V, ml["router"]["top"])
            for e in range(ml["router"]["experts"]):
                shapes.update({f"{p}.mlp.e{e}.gate": (F, W), f"{p}.mlp.e{e}.up": (F, W), f"{p}.mlp.e{e}.down": (W, F)})
    return shapes


def make_weights(c: dict, seed: int) -> dict:
    """Random float32 weights: matrices N(0, 1.5/sqrt(fan_in)), embedding of order one, stored norm weights N(0, 0.1),
    biases N(0, 0.5), score mixing = the identity plus N(0, 0.5), activation numbers around (1, 0.5, -0.3, 0.2); tables
    of different experts in a row."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(c).items():
        last = name.rsplit(".", 1)[-1]
        if last == "table":
            experts = c["layers"][int(name[1:name.index(".")])]["mlp"]["router"]["experts"]
            out[name] = torch.stack([torch.randperm(experts, generator=g)[:shape[1]] for _ in range(shape[0])]).to(torch.int32)
            continue
        z = torch.randn(shape, generator=g, dtype=torch.float32)
        if name == "embed":
            out[name] = z
        elif last == "talk":
            out[name] = torch.eye(shape[0]) + 0.5 * z
        elif last == "act":
            out[name] = torch.tensor([1.0, 0.5, -0.3, 0.2]) + 0.1 * z
        elif last == "b":
            out[name] = 0.5 * z
        elif len(shape) == 1:
            out[name] = 0.1 * z
        else:
            out[name] = (1.5 / shape[1] ** 0.5) * z
    return out


def stored(weights: dict) -> dict:
    """The values that the folder holds (bfloat16), as float64: both sides compute from the same numbers."""
    return {k: v.to(torch.bfloat16).to(torch.float64) if v.is_floating_point() else v for k, v in weights.items()}


def write_folder(folder, c: dict, weights: dict, dtype=torch.bfloat16) -> Path:
    from safetensors.torch import save_file

    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(c))
    save_file({k: (v.to(dtype) if v.is_floating_point() else v).contiguous() for k, v in weights.items()},
              str(folder / "model.safetensors"))
    return folder
