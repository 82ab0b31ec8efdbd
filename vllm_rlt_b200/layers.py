"""Fused elementwise pieces of a decoder layer around the attention call.

Host-side mirror of `apply_rotary_pos_emb` + `KVCacheManager._write_prepared` as
`OuroAttention.forward` chains them (`vllm_rlt/models/ouro.py:179-186` of the reference) and of
`RMSNorm.forward` with the sandwich residual adds of `OuroDecoderLayer.forward`
(`vllm_rlt/layers/normalization.py:20-23`, `models/ouro.py:217-221`).
"""

from __future__ import annotations

import torch

from . import _capi


def _heads_view(t: torch.Tensor, name: str):
    if t.dim() != 3 or t.stride(2) != 1 or t.stride(1) != t.shape[2]:
        raise ValueError(f"{name} must be [rows, heads, head_dim] with a contiguous [heads, head_dim] tail")


def rope_kv_write(q, k, v, cos, sin, key_cache, value_cache, write_blocks, write_offsets, write_mask=None,
                  active_rows=None):
    """Rotate q and k, write the rotated k and v into their pages, return the rotated q.

    `q`, `k`, `v` may be slices of one fused projection output (any row stride).  `cos`, `sin`:
    `[rows, head_dim]` (or `[rows, 1, head_dim]`) in the model dtype, as `RotaryEmbedding.forward`
    returns them.  `key_cache` / `value_cache` are one layer's `[blocks, block, kv_heads,
    head_dim]` views; the addressing arguments are those of `kv_write`.  The result is bit-identical
    to `q * cos + rotate_half(q) * sin` (and the same for k) on tensors of that dtype.
    """
    _capi.require_cuda(q, k, v, cos, sin, key_cache, value_cache, write_blocks, write_offsets, write_mask,
                       active_rows)
    for name, t in (("q", q), ("k", k), ("v", v)):
        _heads_view(t, name)
    rows, q_heads, head_dim = q.shape
    kv_heads = k.shape[1]
    if k.shape != (rows, kv_heads, head_dim) or v.shape != k.shape or head_dim % 2:
        raise ValueError("k and v must be [rows, kv_heads, head_dim] with an even head_dim")
    if not (q.dtype == k.dtype == v.dtype == key_cache.dtype == value_cache.dtype) or q.dtype not in _capi.DTYPE_CODES:
        raise ValueError("q, k, v and the cache must share one of float32 / float16 / bfloat16")
    cos, sin = cos.reshape(rows, head_dim), sin.reshape(rows, head_dim)
    if cos.dtype != q.dtype or sin.dtype != q.dtype:
        raise ValueError("cos and sin must have the model dtype")
    if key_cache.dim() != 4 or key_cache.shape[2:] != (kv_heads, head_dim) or key_cache.stride(3) != 1 \
            or key_cache.stride(2) != head_dim or key_cache.stride() != value_cache.stride() \
            or key_cache.shape != value_cache.shape:
        raise ValueError("cache views must be [blocks, block, kv_heads, head_dim] with equal strides")
    for name, t in (("write_blocks", write_blocks), ("write_offsets", write_offsets)):
        if t.dtype != torch.int64 or t.shape != (rows,):
            raise ValueError(f"{name} must be int64 [rows]")
    mask = None
    if write_mask is not None:
        if write_mask.shape != (rows,) or write_mask.dtype not in (torch.bool, torch.uint8):
            raise ValueError("write_mask must be bool [rows]")
        mask = write_mask.contiguous().view(torch.uint8)
    if active_rows is not None and (active_rows.dtype != torch.int32 or active_rows.numel() != 1):
        raise ValueError("active_rows must be a 0-dim int32 tensor")
    q_out = torch.empty((rows, q_heads, head_dim), dtype=q.dtype, device=q.device)
    if rows == 0:
        return q_out
    cos, sin = cos.contiguous(), sin.contiguous()
    write_blocks, write_offsets = write_blocks.contiguous(), write_offsets.contiguous()
    with torch.cuda.device(q.device):
        code = _capi.load().rlt_rope_kv_write(
            _capi.ptr(q), q.stride(0), _capi.ptr(k), k.stride(0), _capi.ptr(v), v.stride(0),
            _capi.ptr(cos), _capi.ptr(sin), _capi.ptr(q_out), _capi.ptr(key_cache),
            _capi.ptr(value_cache), key_cache.stride(0), key_cache.stride(1), key_cache.shape[0], key_cache.shape[1],
            q_heads, kv_heads, head_dim, _capi.DTYPE_CODES[q.dtype], _capi.ptr(write_blocks),
            _capi.ptr(write_offsets), _capi.ptr(mask), _capi.ptr(active_rows), rows, _capi.stream_of(q))
    _capi.check(code, "rope_kv_write")
    return q_out


def sandwich_norm(x, weight, eps: float, residual=None, weight2=None, *, in_place: bool = False):
    """`total = [residual +] weight * rmsnorm(x)` and, with `weight2`, `norm = weight2 * rmsnorm(total)`.

    Returns `(total, norm)` (`norm` is None without `weight2`).  `in_place` writes `total` over
    `residual` (the residual stream of a decoder layer).  Roundings are those of the tensor
    expressions in the model dtype; the mean of squares is accumulated in double.
    """
    _capi.require_cuda(x, weight, residual, weight2)
    if x.dim() != 2 or not x.is_contiguous() or x.dtype not in _capi.DTYPE_CODES:
        raise ValueError("x must be contiguous [rows, hidden] float32 / float16 / bfloat16")
    rows, hidden = x.shape
    for name, w in (("weight", weight), ("weight2", weight2)):
        if w is not None and (w.shape != (hidden,) or w.dtype != x.dtype or not w.is_contiguous()):
            raise ValueError(f"{name} must be contiguous [hidden] of x's dtype")
    if residual is not None and (residual.shape != x.shape or residual.dtype != x.dtype or not residual.is_contiguous()):
        raise ValueError("residual must match x")
    if in_place and residual is None:
        raise ValueError("in_place needs a residual")
    total = residual if in_place else torch.empty_like(x)
    norm = None if weight2 is None else torch.empty_like(x)
    if rows == 0:
        return total, norm
    with torch.cuda.device(x.device):
        code = _capi.load().rlt_sandwich_norm(_capi.ptr(x), _capi.ptr(weight), _capi.ptr(residual), _capi.ptr(total),
                                              _capi.ptr(weight2), _capi.ptr(norm), rows, hidden, float(eps),
                                              _capi.DTYPE_CODES[x.dtype], _capi.stream_of(x))
    _capi.check(code, "sandwich_norm")
    return total, norm


ACTIVATIONS = {"gelu": 1, "gelu_tanh": 2, "silu": 3, "squared_relu": 4}      # gelu: the erf form


def residual_norm(residual, weight, eps: float, dtype, *, delta=None, tokens=None, embed=None, row_index=None,
                  weight_offset: float = 0.0, store: bool = True, behind=None, centred: bool = False, parts=None):
    """The 32-bit residual stream and the norm that opens a layer or sublayer, in one pass:

        r = embed[tokens] or residual;  r += delta;  residual <- r (with `store`)
        returns norm(r) * (weight_offset + weight), in `dtype`

    norm(r) = r / sqrt(mean(r^2) + eps), with `centred` (a layer norm) of r minus its mean.  behind = (weight, scale): the sublayer has a
    norm behind it too, r += scale * norm(delta) * weight.  parts = (values, rows, weights): the weighted sum of rows of
    `values` (rows int32, weights float32, both `[rows, k]`: a token's experts) joins the delta.  weight None: r itself is returned.  residual: float32 [rows, width], updated in place.  `row_index` (int64)
    selects rows: the result has one row per entry, and the residual is not stored.  `weight`: float32 [width]
    (`weight_offset` 1 for weights stored around zero)."""
    delta_weight, delta_scale = behind if behind is not None else (None, 1.0)
    _capi.require_cuda(residual, weight, delta, tokens, embed, row_index, delta_weight, *(parts or ()))
    if residual.dim() != 2 or residual.dtype != torch.float32 or not residual.is_contiguous():
        raise ValueError("residual must be contiguous float32 [rows, width]")
    rows, width = residual.shape
    if weight is not None and (weight.dtype != torch.float32 or weight.shape != (width,) or not weight.is_contiguous()):
        raise ValueError("weight must be contiguous float32 [width]")
    part_values, part_rows, part_weights = parts if parts is not None else (None, None, None)
    k = 0 if parts is None else part_rows.shape[1]
    if parts is not None and (part_values.dtype != dtype or part_values.dim() != 2 or part_values.shape[1] != width or not part_values.is_contiguous()
                              or part_rows.dtype != torch.int32 or part_weights.dtype != torch.float32 or part_rows.shape != (rows, k)
                              or part_weights.shape != (rows, k) or not part_rows.is_contiguous() or not part_weights.is_contiguous()):
        raise ValueError("parts must be contiguous values [n, width] of the model dtype, int32 rows and float32 weights [rows, k]")
    if delta_weight is not None and ((delta is None and parts is None) or delta_weight.dtype != torch.float32 or delta_weight.shape != (width,)
                                     or not delta_weight.is_contiguous()):
        raise ValueError("the norm behind a sublayer needs a delta and a contiguous float32 [width] weight")
    if dtype not in _capi.DTYPE_CODES:
        raise ValueError("dtype must be float32 / float16 / bfloat16")
    if delta is not None and (delta.shape != residual.shape or delta.dtype != dtype or not delta.is_contiguous()):
        raise ValueError("delta must be a contiguous tensor of the model dtype, shaped like the residual")
    if (tokens is None) != (embed is None):
        raise ValueError("tokens and embed go together")
    if tokens is not None and (tokens.dtype != torch.int64 or tokens.shape != (rows,) or embed.dtype != dtype
                               or embed.dim() != 2 or embed.shape[1] != width or not embed.is_contiguous()):
        raise ValueError("tokens must be int64 [rows] and embed contiguous [vocab, width] of the model dtype")
    if row_index is not None:
        if row_index.dtype != torch.int64 or row_index.dim() != 1:
            raise ValueError("row_index must be int64")
        if store:
            raise ValueError("selected rows are not stored: pass store=False")
        row_index = row_index.contiguous()
    count = rows if row_index is None else row_index.numel()
    out = torch.empty(count, width, dtype=dtype, device=residual.device)
    if count == 0:
        return out
    tokens = None if tokens is None else tokens.contiguous()
    with torch.cuda.device(residual.device):
        code = _capi.load().rlt_residual_norm(
            _capi.ptr(residual), _capi.ptr(delta), _capi.ptr(tokens), _capi.ptr(embed), 0 if embed is None else embed.shape[0],
            _capi.ptr(row_index), int(store), _capi.ptr(weight), float(weight_offset), _capi.ptr(delta_weight), float(delta_scale),
            int(centred), _capi.ptr(part_values), _capi.ptr(part_rows), _capi.ptr(part_weights), k, _capi.ptr(out), count, width, float(eps), _capi.DTYPE_CODES[dtype], _capi.stream_of(residual))
    _capi.check(code, "residual_norm")
    return out


def block_epilogue(proj, batch, *, kv=None, act=None):
    """Columns of a stacked projection to where they are needed, in one launch.

    kv = (key column, value column, key cache, value cache): the rows' keys and values into the pages of
    (batch.row_seq, batch.positions); the caches are `[pages, block, kv_heads, dim]` views.
    act = (first column, width, kind, out, out column): `out[:, out column + c] = kind(proj[:, first column + c])`."""
    rows = proj.shape[0]
    if proj.dim() != 2 or proj.stride(1) != 1 or proj.dtype not in _capi.DTYPE_CODES:
        raise ValueError("proj must be [rows, columns] with unit inner stride")
    if rows == 0 or (kv is None and act is None):
        return
    k_col = k_width = v_col = v_width = 0
    key = value = tables = None
    k_strides = v_strides = (0, 0)
    pages = block = width = 0
    if kv is not None:
        k_col, v_col, key, value = kv
        _capi.require_cuda(proj, key, value, batch.row_seq, batch.positions)
        for name, cache in (("key", key), ("value", value)):
            if cache.dim() != 4 or cache.dtype != proj.dtype or cache.stride(3) != 1 or cache.stride(2) != cache.shape[3]:
                raise ValueError(f"the {name} cache must be [pages, block, kv_heads, dim] of the model dtype with a contiguous tail")
        k_width, v_width = key.shape[2] * key.shape[3], value.shape[2] * value.shape[3]
        if k_col + k_width > proj.shape[1] or v_col + v_width > proj.shape[1] or value.shape[:3] != key.shape[:3]:
            raise ValueError("key or value columns lie outside the projection, or the caches do not match")
        k_strides, v_strides = (key.stride(0), key.stride(1)), (value.stride(0), value.stride(1))
        tables = batch.tables[0]
        pages, block, width = key.shape[0], key.shape[1], tables.shape[1]
    act_col = act_width = kind = out_col = out_stride = 0
    out = None
    if act is not None:
        act_col, act_width, name, out, out_col = act
        _capi.require_cuda(proj, out)
        kind = ACTIVATIONS[name]
        if out.dtype != proj.dtype or out.shape[0] != rows or out.stride(1) != 1 or out_col + act_width > out.shape[1] \
                or act_col + act_width > proj.shape[1]:
            raise ValueError("activation columns lie outside the projection or the output")
        out_stride = out.stride(0)
    with torch.cuda.device(proj.device):
        code = _capi.load().rlt_block_epilogue(
            _capi.ptr(proj), proj.stride(0), k_col, k_width, v_col, v_width, _capi.ptr(key), *k_strides, _capi.ptr(value),
            *v_strides, pages, block, _capi.ptr(tables), width, _capi.ptr(None if kv is None else batch.row_seq),
            _capi.ptr(None if kv is None else batch.positions), act_col, act_width, kind, _capi.ptr(out), out_stride, out_col,
            rows, _capi.DTYPE_CODES[proj.dtype], _capi.stream_of(proj))
    _capi.check(code, "block_epilogue")


def stream_mix(streams, weight, eps: float, dtype, *, delta=None, parts=None, ran=None, follows=None, tokens=None, previous=None,
               embed=None, bigram=None, embed_weight=None, row_index=None, weight_offset: float = 0.0, store: bool = True):
    """Hyper-connected residual streams (float32 `[rows, S, width]`, updated in place) between two sublayers:

        x_t <- sum_s mix[s, t] x_s + out[t] * y        ran = (out [S], mix [S, S]) of the sublayer whose output y is
        u = sum_t in[t] x_t                            follows = in [S] of the next one (None: the plain sum)
        returns rmsnorm(u) * (weight_offset + weight), in `dtype`

    y is `delta` `[rows, width]`, or with parts = (rows, weights), both `[rows, k]`, the weighted sum of rows of `delta`.
    With `tokens` the streams start: all of them `rmsnorm(embed[token] + table[bucket]) * embed_weight`, where
    bigram = (table, mul_prev, mul_cur), the table's last row serves first tokens (`previous` < 0, int32 [rows]) and the
    other rows are the buckets of `previous * mul_prev + token * mul_cur`.  `row_index` as in `residual_norm`."""
    _capi.require_cuda(streams, weight, delta, tokens, previous, embed, embed_weight, row_index)
    if streams.dim() != 3 or streams.dtype != torch.float32 or not streams.is_contiguous():
        raise ValueError("streams must be contiguous float32 [rows, streams, width]")
    rows, count, width = streams.shape
    for name, w, shape in (("weight", weight, (width,)), ("embed_weight", embed_weight, (width,)), ("follows", follows, (count,)),
                           ("out", ran[0] if ran else None, (count,)), ("mix", ran[1] if ran else None, (count, count))):
        if w is not None and (w.dtype != torch.float32 or w.shape != shape or not w.is_contiguous()):
            raise ValueError(f"{name} must be contiguous float32 {list(shape)}")
    if dtype not in _capi.DTYPE_CODES or (ran is None) != (delta is None):
        raise ValueError("dtype must be float32 / float16 / bfloat16; delta and ran go together")
    k, part_rows, part_weights = 0, None, None
    if delta is not None:
        if delta.dtype != dtype or delta.dim() != 2 or delta.shape[1] != width or not delta.is_contiguous():
            raise ValueError("delta must be contiguous [rows, width] of the model dtype")
        if parts is not None:
            part_rows, part_weights = parts
            k = part_rows.shape[1]
            if part_rows.dtype != torch.int32 or part_weights.dtype != torch.float32 or part_rows.shape != (rows, k) \
                    or part_weights.shape != (rows, k) or not part_rows.is_contiguous() or not part_weights.is_contiguous():
                raise ValueError("parts must be int32 rows and float32 weights, both contiguous [rows, k]")
        elif delta.shape[0] != rows:
            raise ValueError("delta needs one row per row of the streams")
    table, buckets, mul_prev, mul_cur = None, 0, 0, 0
    if tokens is not None:
        if tokens.dtype != torch.int64 or tokens.shape != (rows,) or embed is None or embed.dtype != dtype or embed.dim() != 2 \
                or embed.shape[1] != width or not embed.is_contiguous() or embed_weight is None:
            raise ValueError("tokens must be int64 [rows], embed contiguous [vocab, width] of the model dtype, with a norm weight")
        if bigram is not None:
            table, mul_prev, mul_cur = bigram
            buckets = table.shape[0] - 1
            if table.dtype != dtype or table.dim() != 2 or table.shape[1] != width or not table.is_contiguous() or buckets < 1 \
                    or previous is None or previous.dtype != torch.int32 or previous.shape != (rows,):
                raise ValueError("the bigram table must be contiguous [buckets + 1, width] of the model dtype, previous int32 [rows]")
    if row_index is not None:
        if row_index.dtype != torch.int64 or row_index.dim() != 1 or store:
            raise ValueError("row_index must be int64, and selected rows are not stored: pass store=False")
        row_index = row_index.contiguous()
    n = rows if row_index is None else row_index.numel()
    out = torch.empty(n, width, dtype=dtype, device=streams.device)
    if n == 0:
        return out
    with torch.cuda.device(streams.device):
        code = _capi.load().rlt_stream_mix(
            _capi.ptr(streams), count, _capi.ptr(delta), k, _capi.ptr(part_rows), _capi.ptr(part_weights),
            _capi.ptr(ran[0] if ran else None), _capi.ptr(ran[1] if ran else None), _capi.ptr(tokens), _capi.ptr(previous),
            _capi.ptr(embed), 0 if embed is None else embed.shape[0], _capi.ptr(table), buckets, int(mul_prev), int(mul_cur),
            _capi.ptr(embed_weight), _capi.ptr(follows), _capi.ptr(row_index), int(store), _capi.ptr(weight), float(weight_offset),
            _capi.ptr(out), n, width, float(eps), _capi.DTYPE_CODES[dtype], _capi.stream_of(streams))
    _capi.check(code, "stream_mix")
    return out


def clamped_glu(gate_up, up_col: int, cols: int, limit: float, slope: float):
    """`g * sigmoid(slope * g) * (u + 1)` with g = min(gate, limit), u = clamp(up, -limit, limit), over columns 0 .. and
    `up_col` .. of one projection output; returns contiguous `[rows, cols]`."""
    _capi.require_cuda(gate_up)
    if gate_up.dim() != 2 or gate_up.stride(1) != 1 or gate_up.dtype not in _capi.DTYPE_CODES or up_col + cols > gate_up.shape[1]:
        raise ValueError("gate_up must be [rows, columns] with unit inner stride that holds both halves")
    out = torch.empty(gate_up.shape[0], cols, dtype=gate_up.dtype, device=gate_up.device)
    with torch.cuda.device(gate_up.device):
        code = _capi.load().rlt_clamped_glu(_capi.ptr(gate_up), gate_up.stride(0), up_col, _capi.ptr(out), out.stride(0), out.shape[0],
                                            cols, float(limit), float(slope), _capi.DTYPE_CODES[gate_up.dtype], _capi.stream_of(gate_up))
    _capi.check(code, "clamped_glu")
    return out


def gated_unit(gate_up, up_col: int, cols: int, act: str):
    """`act(gate) * up` over columns 0 .. and `up_col` .. of one projection output; returns contiguous `[rows, cols]`."""
    _capi.require_cuda(gate_up)
    if gate_up.dim() != 2 or gate_up.stride(1) != 1 or gate_up.dtype not in _capi.DTYPE_CODES or up_col + cols > gate_up.shape[1]:
        raise ValueError("gate_up must be [rows, columns] with unit inner stride that holds both halves")
    out = torch.empty(gate_up.shape[0], cols, dtype=gate_up.dtype, device=gate_up.device)
    with torch.cuda.device(gate_up.device):
        code = _capi.load().rlt_gated_unit(_capi.ptr(gate_up), gate_up.stride(0), up_col, _capi.ptr(out), out.stride(0), out.shape[0],
                                           cols, ACTIVATIONS[act], _capi.DTYPE_CODES[gate_up.dtype], _capi.stream_of(gate_up))
    _capi.check(code, "gated_unit")
    return out


def check_gate(gate, rows: int, heads: int, dim: int) -> None:
    if gate is not None and gate.shape not in ((rows, heads * dim), (rows, heads)):
        raise ValueError("gate must be [rows, heads * dim] or [rows, heads]")


def per_head(gate, heads: int, dim: int) -> bool:
    """Whether a gate has one value per head and not one per element (with heads of one element both are the same)."""
    return gate.shape[1] == heads and dim != 1


def head_gate(y, gate, out=None):
    """`y * sigmoid(gate)`: y `[rows, heads, dim]` with heads side by side, gate `[rows, heads * dim]` or `[rows, heads]`; out None: in place."""
    out = y if out is None else out
    _capi.require_cuda(y, gate, out)
    rows, heads, dim = y.shape
    check_gate(gate, rows, heads, dim)
    if out.shape != y.shape or any(t.stride(2) != 1 or t.stride(1) != dim for t in (y, out)) or gate.stride(1) != 1 \
            or y.dtype not in _capi.DTYPE_CODES or gate.dtype != y.dtype or out.dtype != y.dtype:
        raise ValueError("y and out must be [rows, heads, dim] with heads side by side, gate of the same dtype with unit inner stride")
    if rows == 0:
        return out
    with torch.cuda.device(y.device):
        code = _capi.load().rlt_head_gate(_capi.ptr(y), y.stride(0), _capi.ptr(gate), gate.stride(0), _capi.ptr(out), out.stride(0), rows, heads,
                                          dim, int(per_head(gate, heads, dim)), _capi.DTYPE_CODES[y.dtype], _capi.stream_of(y))
    _capi.check(code, "head_gate")
    return out


def norm_rotate(proj, columns, q_weight, k_weight, eps: float, frequencies, q_out, key_cache, value_cache, batch, *, halves: bool = False):
    """What stands between an attention layer's projections and its scores: q and k of every head divided by their root mean square times
    their weight (float32 `[dim]`, None: no norm), their first dimensions turned by the position as in `rotate_heads`, k and v into the
    pages of their positions, q into q_out.

    proj `[rows, columns]` holds q, k and v from the three `columns` on; q_out `[rows, heads, dim]`; the caches `[pages, block, kv_heads, dim]`
    views; frequencies float64 (an empty tensor: no rotation)."""
    _capi.require_cuda(proj, q_weight, k_weight, frequencies, q_out, key_cache, value_cache, batch.row_seq, batch.positions)
    rows, heads, key_dim = q_out.shape
    kv_heads, value_dim = value_cache.shape[2], value_cache.shape[3]
    if proj.dim() != 2 or proj.shape[0] != rows or proj.stride(1) != 1 or proj.dtype not in _capi.DTYPE_CODES \
            or any(t.dtype != proj.dtype for t in (q_out, key_cache, value_cache)):
        raise ValueError("proj must be [rows, columns] with unit inner stride; q_out and caches of its dtype")
    if key_cache.shape != (*value_cache.shape[:3], key_dim) or any(c.stride(3) != 1 or c.stride(2) != c.shape[3] for c in (key_cache, value_cache)):
        raise ValueError("caches must be [pages, block, kv_heads, dim] with a contiguous tail, keys as wide as queries")
    if any(at + n > proj.shape[1] for at, n in zip(columns, (heads * key_dim, kv_heads * key_dim, kv_heads * value_dim))):
        raise ValueError("q, k and v must lie in the projection")
    for w in (q_weight, k_weight):
        if w is not None and (w.dtype != torch.float32 or w.shape != (key_dim,) or not w.is_contiguous()):
            raise ValueError("weights must be contiguous float32 [dim]")
    if frequencies.dtype != torch.float64 or 2 * frequencies.numel() > key_dim or q_out.stride(2) != 1 or q_out.stride(1) != key_dim:
        raise ValueError("frequencies must be float64 of at most dim / 2 pairs, q_out [rows, heads, dim] with heads side by side")
    if rows == 0:
        return q_out
    tables = batch.tables[0]
    with torch.cuda.device(proj.device):
        code = _capi.load().rlt_norm_rotate(
            _capi.ptr(proj), proj.stride(0), *columns, heads, kv_heads, key_dim, value_dim, _capi.ptr(q_weight), _capi.ptr(k_weight), float(eps),
            _capi.ptr(frequencies), 2 * frequencies.numel(), int(halves), _capi.ptr(batch.row_seq), _capi.ptr(batch.positions), _capi.ptr(q_out),
            q_out.stride(0), _capi.ptr(key_cache), key_cache.stride(0), key_cache.stride(1), _capi.ptr(value_cache), value_cache.stride(0),
            value_cache.stride(1), key_cache.shape[0], key_cache.shape[1], _capi.ptr(tables), tables.shape[1], rows,
            _capi.DTYPE_CODES[proj.dtype], _capi.stream_of(proj))
    _capi.check(code, "norm_rotate")
    return q_out


def head_mix(y, talk, out, kv_heads: int):
    """`out[:, h] = sum_g talk[h, g] * y[:, g, c(h)]`: y `[rows, heads, kv_heads * dim]` (every head over the values of every key/value head),
    talk float32 `[heads, heads]`, out `[rows, heads, dim]`, c(h) = h // (heads // kv_heads)."""
    _capi.require_cuda(y, talk, out)
    rows, heads, dim = out.shape
    if y.shape != (rows, heads, kv_heads * dim) or any(t.stride(2) != 1 or t.stride(1) != t.shape[2] for t in (y, out)) \
            or y.dtype not in _capi.DTYPE_CODES or out.dtype != y.dtype:
        raise ValueError("y must be [rows, heads, kv_heads * dim] and out [rows, heads, dim] of one dtype, heads side by side")
    if talk.dtype != torch.float32 or talk.shape != (heads, heads) or not talk.is_contiguous() or heads % kv_heads:
        raise ValueError("talk must be contiguous float32 [heads, heads], heads a multiple of kv_heads")
    if rows == 0:
        return out
    with torch.cuda.device(y.device):
        code = _capi.load().rlt_head_mix(_capi.ptr(y), y.stride(0), _capi.ptr(talk), _capi.ptr(out), out.stride(0), rows, heads, kv_heads, dim,
                                         _capi.DTYPE_CODES[y.dtype], _capi.stream_of(y))
    _capi.check(code, "head_mix")
    return out


def soft_cap(x, cap: float):
    """`cap * tanh(x / cap)` of a contiguous float32 tensor, in place."""
    _capi.require_cuda(x)
    if x.dtype != torch.float32 or not x.is_contiguous():
        raise ValueError("x must be contiguous float32")
    with torch.cuda.device(x.device):
        code = _capi.load().rlt_soft_cap(_capi.ptr(x), x.numel(), float(cap), _capi.stream_of(x))
    _capi.check(code, "soft_cap")
    return x
