"""Rows of latent attention: down projections into cache rows, rotation, gathering what a prompt expands (`csrc/latent_rows.cu`)."""

from __future__ import annotations

import math
from dataclasses import dataclass

import torch

from . import _capi
from .attention import check_sink
from .layers import check_gate, per_head


@dataclass(frozen=True)
class YarnScaling:
    """Rotation stretched to `factor` times its original length, after the YaRN paper (Peng, Quesnelle, Fan and Shippole): pairs that make
    more than `fast` turns over the `original` length keep their frequency, those that make fewer than `slow` have it divided by the
    factor, with a linear ramp over the pairs in between; the turned pairs are multiplied by `amplitude`."""

    factor: float
    original: float
    fast: float
    slow: float

    @property
    def amplitude(self) -> float:
        return 0.1 * math.log(self.factor) + 1.0

    def apply(self, frequencies: list, base: float, dims: int) -> list:
        pair = lambda turns: dims * math.log(self.original / (2 * math.pi * turns)) / (2 * math.log(base))
        low, high = max(math.floor(pair(self.fast)), 0), min(math.ceil(pair(self.slow)), dims - 1)
        ramp = [min(max((i - low) / max(high - low, 0.001), 0.0), 1.0) for i in range(len(frequencies))]
        return [f / self.factor * r + f * (1.0 - r) for f, r in zip(frequencies, ramp)]


def rotation_frequencies(base: float, dims: int, device, scaling: YarnScaling | None = None) -> torch.Tensor:
    """base^(-2i / dims) of pair i (with `scaling`: scaled), in float64 (angles are formed and reduced in it)."""
    frequencies = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is not None:
        frequencies = scaling.apply(frequencies, float(base), dims)
    return torch.tensor(frequencies, dtype=torch.float64, device=device)


def latent_write(proj, q_col: int, kv_col: int, q_weight, kv_weight, eps: float, frequencies, cache, batch, *,
                 halves: bool = False, amplitude: float = 1.0):
    """The stacked down projections of a step's rows: returns the normed query latent `[rows, q_rank]` and writes the normed
    key/value latent and the rotated key part (as `rotate_heads` turns), side by side, into `cache`
    `[pages, block, 1, kv_rank + rot_dim]`."""
    _capi.require_cuda(proj, q_weight, kv_weight, frequencies, cache, batch.row_seq, batch.positions)
    rows, q_rank, kv_rank = proj.shape[0], q_weight.numel(), kv_weight.numel()
    if proj.dim() != 2 or proj.stride(1) != 1 or proj.dtype not in _capi.DTYPE_CODES or cache.dtype != proj.dtype:
        raise ValueError("proj must be [rows, columns] with unit inner stride, of the cache's dtype")
    if cache.dim() != 4 or cache.shape[2] != 1 or cache.stride(3) != 1 or cache.shape[3] < kv_rank:
        raise ValueError("cache must be [pages, block, 1, kv_rank + rot_dim] with unit inner stride")
    rot_dim, rot_dims = cache.shape[3] - kv_rank, 2 * frequencies.numel()
    if q_col + q_rank > proj.shape[1] or kv_col + cache.shape[3] > proj.shape[1] or rot_dims > rot_dim:
        raise ValueError("columns outside the projection, or more turned dimensions than the rotated part has")
    for name, t, dtype in (("q_weight", q_weight, torch.float32), ("kv_weight", kv_weight, torch.float32), ("frequencies", frequencies, torch.float64)):
        if t.dtype != dtype or t.dim() != 1 or not t.is_contiguous():
            raise ValueError(f"{name} must be contiguous one-dimensional {dtype}")
    tables = batch.tables[0]
    q = torch.empty(rows, q_rank, dtype=proj.dtype, device=proj.device)
    with torch.cuda.device(proj.device):
        code = _capi.load().rlt_latent_write(
            _capi.ptr(proj), proj.stride(0), q_col, q_rank, kv_col, kv_rank, rot_dim, rot_dims, _capi.ptr(q_weight), _capi.ptr(kv_weight),
            float(eps), _capi.ptr(frequencies), int(halves), float(amplitude), _capi.ptr(q), q.stride(0), _capi.ptr(cache), cache.stride(0), cache.stride(1),
            cache.shape[0], cache.shape[1], _capi.ptr(tables), tables.shape[1], _capi.ptr(batch.row_seq), _capi.ptr(batch.positions), rows,
            _capi.DTYPE_CODES[proj.dtype], _capi.stream_of(proj))
    _capi.check(code, "latent_write")
    return q


def rotate_heads(src, dst, frequencies, positions, *, halves: bool = False, amplitude: float = 1.0, scale: float = 1.0, scaled_from: int = 0):
    """Pairs (2i, 2i + 1) of every head — with `halves` pairs (i, i + n) of n frequencies — turned by position * frequency_i and
    multiplied by `amplitude`; src and dst `[rows, heads, dim]` with any row and head strides (dst may be src); the dimensions
    behind the turned ones are copied.  Heads from `scaled_from` on are multiplied by `scale`, all of their elements."""
    _capi.require_cuda(src, dst, frequencies, positions)
    rows, heads, dim = src.shape
    if dst.shape != src.shape or dst.dtype != src.dtype or src.stride(2) != 1 or dst.stride(2) != 1 or src.dtype not in _capi.DTYPE_CODES:
        raise ValueError("src and dst must be [rows, heads, dim] of one dtype with unit inner stride")
    if positions.dtype != torch.int32 or positions.shape != (rows,) or frequencies.dtype != torch.float64 or 2 * frequencies.numel() > dim:
        raise ValueError("positions must be int32 [rows], frequencies float64 of at most dim / 2 pairs")
    if rows == 0 or dim == 0:
        return dst
    with torch.cuda.device(src.device):
        code = _capi.load().rlt_rotate_heads(_capi.ptr(src), src.stride(0), src.stride(1), _capi.ptr(dst), dst.stride(0), dst.stride(1), heads,
                                             dim, 2 * frequencies.numel(), _capi.ptr(frequencies), int(halves), float(amplitude),
                                             float(scale), int(scaled_from), _capi.ptr(positions), rows, _capi.DTYPE_CODES[src.dtype], _capi.stream_of(src))
    _capi.check(code, "rotate_heads")
    return dst


def latent_gather(cache, tables, ranges):
    """The cache rows of `ranges` (KeyRanges, with the first tokens it keeps) side by side: `[ranges.rows, row width]`."""
    _capi.require_cuda(cache, tables, ranges.first, ranges.cu)
    if cache.dim() != 4 or cache.shape[2] != 1 or cache.stride(3) != 1 or tables.dtype != torch.int32 or not tables.is_contiguous():
        raise ValueError("cache must be [pages, block, 1, width], tables contiguous int32 [sequences, pages]")
    out = torch.empty(ranges.rows, cache.shape[3], dtype=cache.dtype, device=cache.device)
    with torch.cuda.device(cache.device):
        code = _capi.load().rlt_latent_gather(_capi.ptr(cache), cache.stride(0), cache.stride(1), cache.shape[0], cache.shape[1], cache.shape[3],
                                              _capi.ptr(tables), tables.shape[1], _capi.ptr(ranges.first), _capi.ptr(ranges.cu),
                                              tables.shape[0], ranges.rows, ranges.keep, _capi.ptr(out), _capi.DTYPE_CODES[cache.dtype],
                                              _capi.stream_of(cache))
    _capi.check(code, "latent_gather")
    return out


def latent_prompt_supported(dim: int, rot_dim: int, vdim: int, dtype) -> bool:
    """Whether `latent_prompt_attention` takes heads of these sizes."""
    return bool(_capi.load().rlt_latent_prompt_supported(dim, rot_dim, vdim, _capi.DTYPE_CODES[dtype]))


def packed_attention(q, keys, values, out, ranges, scale: float, window: int, *, shared_keys=None, sink=None, gate=None):
    """Attention of portions over packed keys and values, into `out`; `ranges` (KeyRanges) of the same window.

    q `[rows, heads, dim + rot_dim]`, keys `[ranges.rows, kv_heads, dim]`, values `[ranges.rows, kv_heads, vdim]`, shared_keys
    `[ranges.rows, rot_dim]`: a part of the key that all heads share (None: rot_dim 0); all with any row stride.  out
    `[rows, heads, vdim]`.  sink float32 `[heads]` as in `ScoreTerms`.  gate `[rows, heads * vdim]` or `[rows, heads]`: the output is
    multiplied by its sigmoid, element by element or head by head."""
    _capi.require_cuda(q, keys, values, shared_keys, out, sink, gate, ranges.tiles)
    rows, heads, key_dim = q.shape
    vdim, rot_dim = out.shape[2], 0 if shared_keys is None else shared_keys.shape[1]
    dim, kv_heads = key_dim - rot_dim, keys.shape[1]
    if out.shape[:2] != (rows, heads) or keys.shape != (ranges.rows, kv_heads, dim) or values.shape != (ranges.rows, kv_heads, vdim) \
            or (shared_keys is not None and shared_keys.shape[0] != ranges.rows) or heads % kv_heads:
        raise ValueError("q [rows, heads, dim + rot_dim], out [rows, heads, vdim], one row per packed key, whole groups of heads")
    tensors = [t for t in (q, keys, values, shared_keys, out, gate) if t is not None]
    if any(t.dtype != q.dtype for t in tensors) or any(t.stride(-1) != 1 for t in tensors) \
            or q.stride(1) != key_dim or out.stride(1) != vdim or keys.stride(1) != dim or values.stride(1) != vdim:
        raise ValueError("one dtype, unit inner strides, heads side by side")
    check_sink(sink, heads)
    check_gate(gate, rows, heads, vdim)
    if rows == 0:
        return out
    workspace = torch.empty(256, dtype=torch.uint8, device=q.device)
    with torch.cuda.device(q.device):
        code = _capi.load().rlt_latent_prompt_attention(
            _capi.ptr(q), q.stride(0), _capi.ptr(keys), keys.stride(0), _capi.ptr(values), values.stride(0), _capi.ptr(shared_keys),
            0 if shared_keys is None else shared_keys.stride(0), _capi.ptr(out), out.stride(0), rows, ranges.rows, heads, kv_heads, dim, rot_dim, vdim,
            _capi.ptr(ranges.tiles), ranges.tiles.shape[0], float(scale), int(window), _capi.ptr(sink), _capi.ptr(gate),
            0 if gate is None else gate.stride(0), int(gate is not None and per_head(gate, heads, vdim)), _capi.DTYPE_CODES[q.dtype],
            _capi.ptr(workspace), _capi.stream_of(q))
    _capi.check(code, "latent_prompt_attention")
    return out


def latent_prompt_attention(q, kv, shared_keys, out, dim: int, ranges, scale: float, window: int, *, sink=None, gate=None):
    """`packed_attention` over the one projection that expands latents: kv `[ranges.rows, heads * dim + heads * vdim]` (keys, then
    values, head by head)."""
    heads, vdim = out.shape[1], out.shape[2]
    if kv.shape != (ranges.rows, heads * (dim + vdim)):
        raise ValueError("kv must be [packed keys, heads * dim + heads * vdim]")
    keys, values = kv[:, :heads * dim].unflatten(1, (heads, dim)), kv[:, heads * dim:].unflatten(1, (heads, vdim))
    return packed_attention(q, keys, values, out, ranges, scale, window, shared_keys=shared_keys, sink=sink, gate=gate)
