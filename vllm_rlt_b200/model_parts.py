"""What the model classes of the registry share: reading config entries, stacking projections, GEMM precision."""

from __future__ import annotations

from contextlib import contextmanager

import torch
import torch.nn.functional as F


def take_keys(entry: dict, what: str, required, optional=()) -> dict:
    """The named keys of a config entry; a key nobody knows, unless it is off, is an error and not a guess."""
    missing = [k for k in required if k not in entry]
    if missing:
        raise ValueError(f"{what}: config lacks {missing}")
    unknown = [k for k, v in entry.items() if k not in required and k not in optional and v not in (None, False)]
    if unknown:
        raise ValueError(f"{what}: unknown config keys {unknown}")
    return {k: entry.get(k) for k in (*required, *optional)}


def check_positive(what: str, **sizes) -> None:
    for name, value in sizes.items():
        if isinstance(value, bool) or not isinstance(value, int) or value < 1:
            raise ValueError(f"{what}: {name} must be a positive integer")


def check_shapes(shapes: dict, state_dict: dict) -> None:
    """The state dict holds every parameter in its shape."""
    missing = sorted(set(shapes) - set(state_dict))
    if missing:
        raise ValueError(f"state dict lacks {missing[:3]}{'...' if len(missing) > 3 else ''}")
    for name, shape in shapes.items():
        if tuple(state_dict[name].shape) != shape:
            raise ValueError(f"{name} has shape {tuple(state_dict[name].shape)}, the configuration needs {shape}")


def aligned(columns: int) -> int:
    """Column blocks of a stacked projection start at multiples of 8 elements (16 bytes in 16-bit types)."""
    return -(-columns // 8) * 8


def stack_blocks(blocks, dim: int):
    """Weights side by side along `dim`, each block padded with zeros to a multiple of 8; the blocks' offsets, and the total."""
    parts, offsets, at = [], [], 0
    for block in blocks:
        pad = aligned(block.shape[dim]) - block.shape[dim]
        parts.append(block if not pad else F.pad(block, (0, pad) if dim == 1 else (0, 0, 0, pad)))
        offsets.append(at)
        at += block.shape[dim] + pad
    return torch.cat(parts, dim).contiguous(), offsets, at


@contextmanager
def full_accumulation():
    """fp32 accumulation in every GEMM: no TF32 for 32-bit inputs, no 16-bit partial sums for 16-bit ones."""
    m = torch.backends.cuda.matmul
    saved = m.allow_tf32, m.allow_bf16_reduced_precision_reduction
    m.allow_tf32, m.allow_bf16_reduced_precision_reduction = False, False
    try:
        yield
    finally:
        m.allow_tf32, m.allow_bf16_reduced_precision_reduction = saved


def product32(x, weight):
    """x W^T with an fp32 result."""
    return F.linear(x, weight) if x.dtype == torch.float32 else torch.mm(x, weight.t(), out_dtype=torch.float32)
