"""Random weights for a model, by tensor name.

Each tensor is drawn from its own generator, seeded from (seed, name), so the values do
not depend on the order in which tensors are made or on how parts pack them.  Matrices
and tables of floats are N(0, 0.02); norm weights are 1 + N(0, 0.1); mixing matrices are the identity + N(0, 0.1);
rows of integer tables are different integers below the table's bound.  `write_model_folder`
makes a folder (config.json, model.safetensors) that loads like any other.
"""

from __future__ import annotations

import hashlib
import json
from pathlib import Path

import torch

from ..parts.base import FREE_AXIS

MATRIX_STD = 0.02
NORM_STD = 0.1


def tensor_seed(seed: int, name: str) -> int:
    h = hashlib.sha256(f"{seed}:{name}".encode()).digest()
    return int.from_bytes(h[:8], "little") & ((1 << 63) - 1)


def random_tensor(name: str, spec, seed: int, dtype: torch.dtype, device="cpu") -> torch.Tensor:
    gen = torch.Generator(device=device)
    gen.manual_seed(tensor_seed(seed, name))
    shape = tuple(FREE_AXIS if d == -1 else d for d in spec.shape)
    if spec.kind == "table":
        if not spec.below:
            return torch.zeros(shape, dtype=torch.int32, device=device)
        # the places of the smallest of `below` random numbers: different within a row, every choice equally likely
        keys = torch.rand((shape[0], spec.below), generator=gen, dtype=torch.float32, device=device)
        return keys.argsort(dim=1)[:, :shape[1]].to(torch.int32).contiguous()
    z = torch.randn(shape, generator=gen, dtype=torch.float32, device=device)
    if spec.init == "ones_normal":
        z = 1.0 + NORM_STD * z
    elif spec.init == "eye_normal":
        z = torch.eye(shape[0], shape[1], device=device) + NORM_STD * z
    else:
        z = MATRIX_STD * z
    return z.to(dtype)


def random_tensors(specs: dict, seed: int, dtype: torch.dtype, device="cpu") -> dict[str, torch.Tensor]:
    return {name: random_tensor(name, spec, seed, dtype, device) for name, spec in specs.items()}


def write_model_folder(folder, config, seed: int, dtype: torch.dtype = torch.bfloat16) -> Path:
    """Writes config.json and model.safetensors for `config` (an architecture's
    configuration object) with random weights stored as `dtype`."""
    from safetensors.torch import save_file

    from ..parts import BuildContext, Model

    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    model = Model(config.to_spec(), BuildContext(dtype=dtype, device=torch.device("cpu")))
    tensors = random_tensors(model.tensor_specs(), seed, dtype, "cpu")
    (folder / "config.json").write_text(json.dumps(config.to_dict(), indent=1))
    save_file({k: v.contiguous() for k, v in tensors.items()}, str(folder / "model.safetensors"))
    return folder
