"""Rows of latent attention: down projections into cache rows, rotation, gathering what a prompt expands (`csrc/latent_rows.cu`)."""

from __future__ import annotations

import torch

from . import _capi


def rotation_frequencies(base: float, dims: int, device) -> torch.Tensor:
    """base^(-2i / dims) of pair i, in float64 (angles are formed and reduced in it)."""
    return torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64, device=device)


def latent_write(proj, q_col: int, kv_col: int, q_weight, kv_weight, eps: float, frequencies, cache, batch):
    """The stacked down projections of a step's rows: returns the normed query latent `[rows, q_rank]` and writes the normed
    key/value latent and the rotated key part, side by side, into `cache` `[pages, block, 1, kv_rank + rot_dim]`."""
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
            float(eps), _capi.ptr(frequencies), _capi.ptr(q), q.stride(0), _capi.ptr(cache), cache.stride(0), cache.stride(1),
            cache.shape[0], cache.shape[1], _capi.ptr(tables), tables.shape[1], _capi.ptr(batch.row_seq), _capi.ptr(batch.positions), rows,
            _capi.DTYPE_CODES[proj.dtype], _capi.stream_of(proj))
    _capi.check(code, "latent_write")
    return q


def rotate_heads(src, dst, frequencies, positions):
    """Pairs (2i, 2i + 1) of every head turned by position * frequency_i; src and dst `[rows, heads, dim]` with any row and
    head strides (dst may be src); the dimensions behind the turned ones are copied."""
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
                                             dim, 2 * frequencies.numel(), _capi.ptr(frequencies), _capi.ptr(positions), rows,
                                             _capi.DTYPE_CODES[src.dtype], _capi.stream_of(src))
    _capi.check(code, "rotate_heads")
    return dst


def latent_gather(cache, tables, ranges):
    """The cache rows of `ranges` (KeyRanges) side by side: `[ranges.rows, row width]`."""
    _capi.require_cuda(cache, tables, ranges.first, ranges.cu)
    if cache.dim() != 4 or cache.shape[2] != 1 or cache.stride(3) != 1 or tables.dtype != torch.int32 or not tables.is_contiguous():
        raise ValueError("cache must be [pages, block, 1, width], tables contiguous int32 [sequences, pages]")
    out = torch.empty(ranges.rows, cache.shape[3], dtype=cache.dtype, device=cache.device)
    with torch.cuda.device(cache.device):
        code = _capi.load().rlt_latent_gather(_capi.ptr(cache), cache.stride(0), cache.stride(1), cache.shape[0], cache.shape[1], cache.shape[3],
                                              _capi.ptr(tables), tables.shape[1], _capi.ptr(ranges.first), _capi.ptr(ranges.cu),
                                              tables.shape[0], ranges.rows, _capi.ptr(out), _capi.DTYPE_CODES[cache.dtype],
                                              _capi.stream_of(cache))
    _capi.check(code, "latent_gather")
    return out


def latent_prompt_supported(dim: int, rot_dim: int, vdim: int, dtype) -> bool:
    """Whether `latent_prompt_attention` takes heads of these sizes."""
    return bool(_capi.load().rlt_latent_prompt_supported(dim, rot_dim, vdim, _capi.DTYPE_CODES[dtype]))


def latent_prompt_attention(q, kv, shared_keys, out, dim: int, ranges, scale: float, window: int):
    """Attention of portions over packed keys and values expanded from latents, into `out`.

    q `[rows, heads, dim + rot_dim]`, kv `[ranges.rows, heads * dim + heads * vdim]` (keys, then values, head by head),
    shared_keys `[ranges.rows, rot_dim]` (any row stride), out `[rows, heads, vdim]`; `ranges` (KeyRanges) of the same window."""
    _capi.require_cuda(q, kv, shared_keys, out, ranges.tiles)
    rows, heads, key_dim = q.shape
    vdim, rot_dim = out.shape[2], key_dim - dim
    if out.shape[:2] != (rows, heads) or kv.shape != (ranges.rows, heads * (dim + vdim)) or shared_keys.shape != (ranges.rows, rot_dim):
        raise ValueError("q [rows, heads, dim + rot_dim], out [rows, heads, vdim], kv and shared_keys one row per packed key")
    if any(t.dtype != q.dtype for t in (kv, shared_keys, out)) or any(t.stride(-1) != 1 for t in (q, kv, shared_keys, out)) \
            or q.stride(1) != key_dim or out.stride(1) != vdim:
        raise ValueError("one dtype, unit inner strides, heads side by side")
    if rows == 0:
        return out
    workspace = torch.empty(256, dtype=torch.uint8, device=q.device)
    with torch.cuda.device(q.device):
        code = _capi.load().rlt_latent_prompt_attention(
            _capi.ptr(q), q.stride(0), _capi.ptr(kv), kv.stride(0), _capi.ptr(shared_keys), shared_keys.stride(0), _capi.ptr(out), out.stride(0),
            rows, ranges.rows, heads, dim, rot_dim, vdim, _capi.ptr(ranges.tiles), ranges.tiles.shape[0], float(scale), int(window),
            _capi.DTYPE_CODES[q.dtype], _capi.ptr(workspace), _capi.stream_of(q))
    _capi.check(code, "latent_prompt_attention")
    return out
