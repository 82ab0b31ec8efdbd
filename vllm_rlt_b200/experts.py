"""Mixture-of-experts feed-forward: routing, rows sorted by expert, grouped products (`csrc/experts.cu`)."""

from __future__ import annotations

from dataclasses import dataclass

import torch

from . import _capi
from .layers import ACTIVATIONS


@dataclass
class Routing:
    counts: torch.Tensor     # int32 [experts], rows of every expert
    chosen: torch.Tensor     # int32 [rows, top]
    rank: torch.Tensor       # int32 [rows, top], place in the chosen expert's queue
    weights: torch.Tensor    # float32 [rows, top]
    places: torch.Tensor     # int32 [rows, top], row of each choice among the sorted rows


def expert_route(logits, correction, top: int, *, bias=None, counts=None, floor_sum: float = 1e-20) -> Routing:
    """s = softmax(logits + bias) in fp32 (bias float32 [experts] or None); the `top` largest of s + correction (float32 [experts], None: of
    the logits) are chosen, weighted by their s over the sum of the chosen s + floor_sum (0: the softmax over the chosen logits alone).  `counts`: int32 [experts] of zeros (None: allocated)."""
    _capi.require_cuda(logits, correction, bias, counts)
    rows, experts = logits.shape
    if logits.dtype != torch.float32 or logits.stride(1) != 1:
        raise ValueError("logits must be float32 [rows, experts]")
    for name, t in (("correction", correction), ("bias", bias)):
        if t is not None and (t.dtype != torch.float32 or t.shape != (experts,)):
            raise ValueError(f"{name} must be float32 [experts]")
    if counts is None:
        counts = torch.zeros(experts, dtype=torch.int32, device=logits.device)
    elif counts.dtype != torch.int32 or counts.shape != (experts,) or not counts.is_contiguous():
        raise ValueError("counts must be contiguous int32 [experts]")
    slots = torch.empty(3, rows, top, dtype=torch.int32, device=logits.device)
    weights = torch.empty(rows, top, dtype=torch.float32, device=logits.device)
    with torch.cuda.device(logits.device):
        code = _capi.load().rlt_expert_route(_capi.ptr(logits), logits.stride(0), _capi.ptr(bias), _capi.ptr(correction), rows, experts, top, float(floor_sum),
                                             _capi.ptr(counts), _capi.ptr(slots[0]), _capi.ptr(slots[1]), _capi.ptr(weights),
                                             _capi.stream_of(logits))
    _capi.check(code, "expert_route")
    return Routing(counts, slots[0], slots[1], weights, slots[2])


def expert_gather(x, routing: Routing):
    """The rows sorted by expert, `[rows * top, width]`; fills `routing.places`."""
    _capi.require_cuda(x, routing.chosen)
    rows, width = x.shape
    top = routing.chosen.shape[1]
    if x.stride(1) != 1 or x.dtype not in _capi.DTYPE_CODES or routing.chosen.shape[0] != rows:
        raise ValueError("x must be [rows, width] with unit inner stride, one row per routed row")
    out = torch.empty(rows * top, width, dtype=x.dtype, device=x.device)
    with torch.cuda.device(x.device):
        code = _capi.load().rlt_expert_gather(_capi.ptr(x), x.stride(0), _capi.ptr(routing.counts), _capi.ptr(routing.chosen),
                                              _capi.ptr(routing.rank), rows, top, width, _capi.ptr(out), _capi.ptr(routing.places),
                                              _capi.DTYPE_CODES[x.dtype], _capi.stream_of(x))
    _capi.check(code, "expert_gather")
    return out


def expert_gemm(x, weights, counts, activation: str | None = None, *, paired: bool = False):
    """`act(x W_e^T)` over rows sorted by expert: x `[rows, in]`, weights `[experts, out, in]`, counts int32 `[experts]`.  `paired`: weight
    rows 2i and 2i + 1 are a gate and what it multiplies (`paired_rows`), the result is `act(gate) * up`, `[rows, out / 2]`."""
    _capi.require_cuda(x, weights, counts)
    experts, out_width, in_width = weights.shape
    if x.dim() != 2 or x.shape[1] != in_width or x.stride(1) != 1 or x.dtype not in _capi.DTYPE_CODES or weights.dtype != x.dtype \
            or not weights.is_contiguous() or counts.dtype != torch.int32 or counts.shape != (experts,):
        raise ValueError("x [rows, in] and contiguous weights [experts, out, in] of one dtype, counts int32 [experts]")
    if paired and (out_width % 2 or not activation):
        raise ValueError("paired weights need an even number of rows and an activation")
    y = torch.empty(x.shape[0], out_width // 2 if paired else out_width, dtype=x.dtype, device=x.device)
    workspace = torch.empty(256, dtype=torch.uint8, device=x.device)
    with torch.cuda.device(x.device):
        code = _capi.load().rlt_expert_gemm(_capi.ptr(x), x.stride(0), _capi.ptr(weights), _capi.ptr(y), y.stride(0), _capi.ptr(counts),
                                            x.shape[0], experts, in_width, out_width, ACTIVATIONS[activation] if activation else 0, int(paired),
                                            _capi.DTYPE_CODES[x.dtype], _capi.ptr(workspace), _capi.stream_of(x))
    _capi.check(code, "expert_gemm")
    return y


def paired_rows(gate, up):
    """The rows of two weights `[.., out, in]` in turn, as `expert_gemm(paired=True)` takes them."""
    return torch.stack([gate, up], -2).flatten(-3, -2).contiguous()
