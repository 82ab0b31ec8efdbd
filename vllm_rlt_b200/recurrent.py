"""Recurrent layers over packed sequences with per-sequence state slots: short causal convolution (also as part of what prepares
an attention layer's heads), the Mamba-2 state-space recurrence, linear attention with constant decays, the gated delta rule, and the gated norm behind them.

`group` arguments are a step's sequence group (`StepGroup`): `cu` (int32 [n + 1], row offsets into the step's
rows), `starts` (position of each portion's first token), `slots`, and the host-side bound `max_new`.
"""

from __future__ import annotations

import torch

from . import _capi
from .layers import ACTIVATIONS


def causal_conv(x, weight, bias, state, out, group, act=None):
    """`out[i, c] = silu(bias[c] + sum_j weight[c, j] * x[i - taps + 1 + j, c])`, inputs before a portion from `state`.

    x `[rows, channels]` (any row stride), weight float32 `[channels, taps]`, bias float32 `[channels]`, state
    `[slots, taps - 1, channels]` of x's dtype, updated in place.  act = (columns, kind, destination): feed-forward
    columns of the same rows through an activation in the same launch."""
    device = _capi.require_cuda(x, weight, bias, state, out, group.cu, group.starts, group.slots)
    channels, taps = weight.shape
    if weight.dtype != torch.float32 or bias.dtype != torch.float32 or bias.shape != (channels,) or not weight.is_contiguous():
        raise ValueError("weight must be contiguous float32 [channels, taps] and bias float32 [channels]")
    if x.dim() != 2 or x.shape[1] != channels or out.shape != x.shape or x.stride(1) != 1 or out.stride(1) != 1 \
            or x.dtype not in _capi.DTYPE_CODES or out.dtype != x.dtype:
        raise ValueError("x and out must be [rows, channels] of one dtype with unit inner stride")
    if state.shape[1:] != (taps - 1, channels) or state.dtype != x.dtype or not state.is_contiguous():
        raise ValueError("state must be contiguous [slots, taps - 1, channels] of the model dtype")
    act_in, act_out, act_width, kind = None, None, 0, 0
    if act is not None:
        act_in, name, act_out = act
        kind, act_width = ACTIVATIONS[name], act_in.shape[1]
        if act_in.stride(0) != x.stride(0) or act_in.stride(1) != 1 or act_out.shape != act_in.shape or act_out.stride(1) != 1 \
                or act_in.dtype != x.dtype or act_out.dtype != x.dtype:
            raise ValueError("activation columns must come from the projection that holds x")
    if group.sequences == 0:
        return out
    with torch.cuda.device(device):
        code = _capi.load().rlt_causal_conv(
            _capi.ptr(x), x.stride(0), _capi.ptr(weight), _capi.ptr(bias), _capi.ptr(out), out.stride(0), _capi.ptr(state),
            state.shape[0], channels, taps, _capi.ptr(group.cu), _capi.ptr(group.starts), _capi.ptr(group.slots), group.sequences,
            group.max_new, _capi.ptr(act_in), _capi.ptr(act_out), 0 if act_out is None else act_out.stride(0), act_width, kind,
            _capi.DTYPE_CODES[x.dtype], _capi.stream_of(x))
    _capi.check(code, "causal_conv")
    return out


def conv_heads(proj, columns, weight, eps: float, state, q_out, key_cache, value_cache, group, *, unit_norm: bool = True):
    """What stands between an attention layer's projections and its scores: `out[i, c] = sum_j weight[j, c] * x[i - taps + 1 + j, c]`
    over the channels of q, k and v, with `unit_norm` q and k of every head divided by their root mean square, k and v into the pages of
    their positions, q into q_out.

    proj `[rows, columns]` holds q, k and v from the three `columns` on; weight float32 `[taps, channels]` (channels in the order q, k, v);
    state `[slots, taps - 1, channels]` of proj's dtype, updated in place; q_out `[rows, heads, dim]`; the caches
    `[pages, block, kv_heads, dim]` views."""
    device = _capi.require_cuda(proj, weight, state, q_out, key_cache, value_cache, group.cu, group.starts, group.slots, group.lengths, group.tables)
    rows, heads, key_dim = q_out.shape
    kv_heads, value_dim = value_cache.shape[2], value_cache.shape[3]
    taps, channels = weight.shape
    if proj.dim() != 2 or proj.shape[0] != rows or proj.stride(1) != 1 or proj.dtype not in _capi.DTYPE_CODES \
            or any(t.dtype != proj.dtype for t in (state, q_out, key_cache, value_cache)):
        raise ValueError("proj must be [rows, columns] with unit inner stride; state, q_out and caches of its dtype")
    if key_cache.shape != (*value_cache.shape[:3], key_dim) or any(c.stride(3) != 1 or c.stride(2) != c.shape[3] for c in (key_cache, value_cache)):
        raise ValueError("caches must be [pages, block, kv_heads, dim] with a contiguous tail, keys as wide as queries")
    widths = heads * key_dim, kv_heads * key_dim, kv_heads * value_dim
    if channels != sum(widths) or any(at + n > proj.shape[1] for at, n in zip(columns, widths)):
        raise ValueError("weight needs a column per channel of q, k and v; their columns must lie in the projection")
    if weight.dtype != torch.float32 or not weight.is_contiguous() or state.shape[1:] != (taps - 1, channels) or not state.is_contiguous():
        raise ValueError("weight must be contiguous float32 [taps, channels], state contiguous [slots, taps - 1, channels]")
    if q_out.stride(2) != 1 or q_out.stride(1) != key_dim:
        raise ValueError("q_out must be [rows, heads, dim] with heads side by side")
    if group.sequences == 0:
        return q_out
    with torch.cuda.device(device):
        code = _capi.load().rlt_conv_heads(
            _capi.ptr(proj), proj.stride(0), *columns, heads, kv_heads, key_dim, value_dim, _capi.ptr(weight), taps, int(unit_norm), float(eps),
            _capi.ptr(state), state.shape[0], _capi.ptr(q_out), q_out.stride(0), _capi.ptr(key_cache), key_cache.stride(0), key_cache.stride(1),
            _capi.ptr(value_cache), value_cache.stride(0), value_cache.stride(1), key_cache.shape[0], key_cache.shape[1], _capi.ptr(group.tables),
            group.tables.shape[1], _capi.ptr(group.cu), _capi.ptr(group.starts), _capi.ptr(group.lengths), _capi.ptr(group.slots), group.sequences,
            group.max_new, _capi.DTYPE_CODES[proj.dtype], _capi.stream_of(proj))
    _capi.check(code, "conv_heads")
    return q_out


def ssd_scan(x, b, c, dt, dt_bias, a_log, d, state, out, group):
    """The Mamba-2 recurrence (`rlt_ssd_scan`): x, out `[rows, heads * head_dim]`, b, c `[rows, groups * state_size]`
    (slices of rows of one stride), dt `[rows, heads]` raw, parameters float32 `[heads]`, state float32
    `[slots, heads, state_size, head_dim]`, updated in place."""
    device = _capi.require_cuda(x, b, c, dt, dt_bias, a_log, d, state, out, group.cu, group.starts, group.slots)
    if state.dim() != 4 or state.dtype != torch.float32 or not state.is_contiguous():
        raise ValueError("state must be contiguous float32 [slots, heads, state_size, head_dim]")
    slots, heads, size, head_dim = state.shape
    rows = x.shape[0]
    if x.shape != (rows, heads * head_dim) or out.shape != x.shape or b.shape != c.shape or b.shape[1] % size or dt.shape != (rows, heads):
        raise ValueError("x / out [rows, heads * head_dim], b / c [rows, groups * state_size], dt [rows, heads]")
    groups = b.shape[1] // size
    if x.stride(0) != b.stride(0) or b.stride(0) != c.stride(0) or any(t.stride(1) != 1 for t in (x, b, c, dt, out)):
        raise ValueError("x, b and c must be column slices of the same rows")
    if x.dtype not in (torch.float32, torch.bfloat16) or any(t.dtype != x.dtype for t in (b, c, dt, out)):
        raise ValueError("x, b, c, dt and out must share float32 or bfloat16")
    for name, t in (("dt_bias", dt_bias), ("a_log", a_log), ("d", d)):
        if t.dtype != torch.float32 or t.shape != (heads,):
            raise ValueError(f"{name} must be float32 [heads]")
    if group.sequences == 0:
        return out
    lib, dtype = _capi.load(), _capi.DTYPE_CODES[x.dtype]
    with torch.cuda.device(device):
        nbytes = lib.rlt_ssd_scan_workspace_bytes(group.sequences, group.max_new, heads, size, head_dim, dtype)
        workspace = torch.empty(nbytes, dtype=torch.uint8, device=device)
        code = lib.rlt_ssd_scan(
            _capi.ptr(x), _capi.ptr(b), _capi.ptr(c), x.stride(0), _capi.ptr(dt), dt.stride(0), _capi.ptr(dt_bias),
            _capi.ptr(a_log), _capi.ptr(d), _capi.ptr(out), out.stride(0), _capi.ptr(state), slots, _capi.ptr(group.cu),
            _capi.ptr(group.starts), _capi.ptr(group.slots), group.sequences, group.max_new, heads, groups, size, head_dim, dtype,
            _capi.ptr(workspace), nbytes, _capi.stream_of(x))
    _capi.check(code, "ssd_scan")
    return out


def decay_scan(q, k, v, decay, state, out, group):
    """Linear attention with a constant decay per head (`rlt_decay_scan`): `S_t = decay S_(t-1) + k_t v_t^T`, `out_t = S_t^T q_t`.

    q, k `[rows, heads * key_dim]`, v, out `[rows, heads * value_dim]` (q, k and v slices of rows of one stride), decay float32
    `[2, heads]` (`decay_table`), state float32 `[slots, heads, key_dim, value_dim]`, updated in place."""
    device = _capi.require_cuda(q, k, v, decay, state, out, group.cu, group.starts, group.slots)
    if state.dim() != 4 or state.dtype != torch.float32 or not state.is_contiguous():
        raise ValueError("state must be contiguous float32 [slots, heads, key_dim, value_dim]")
    slots, heads, key_dim, value_dim = state.shape
    rows = q.shape[0]
    if q.shape != (rows, heads * key_dim) or k.shape != q.shape or v.shape != (rows, heads * value_dim) or out.shape != v.shape:
        raise ValueError("q / k [rows, heads * key_dim], v / out [rows, heads * value_dim]")
    if q.stride(0) != k.stride(0) or k.stride(0) != v.stride(0) or any(t.stride(1) != 1 for t in (q, k, v, out)):
        raise ValueError("q, k and v must be column slices of the same rows")
    if q.dtype not in (torch.float32, torch.bfloat16) or any(t.dtype != q.dtype for t in (k, v, out)):
        raise ValueError("q, k, v and out must share float32 or bfloat16")
    if decay.dtype != torch.float32 or decay.shape != (2, heads) or not decay.is_contiguous():
        raise ValueError("decay must be contiguous float32 [2, heads]")
    if group.sequences == 0:
        return out
    lib, dtype = _capi.load(), _capi.DTYPE_CODES[q.dtype]
    with torch.cuda.device(device):
        nbytes = lib.rlt_ssd_scan_workspace_bytes(group.sequences, group.max_new, heads, key_dim, value_dim, dtype)
        workspace = torch.empty(nbytes, dtype=torch.uint8, device=device)
        code = lib.rlt_decay_scan(
            _capi.ptr(q), _capi.ptr(k), _capi.ptr(v), q.stride(0), _capi.ptr(decay), _capi.ptr(out), out.stride(0), _capi.ptr(state),
            slots, _capi.ptr(group.cu), _capi.ptr(group.starts), _capi.ptr(group.slots), group.sequences, group.max_new, heads, key_dim,
            value_dim, dtype, _capi.ptr(workspace), nbytes, _capi.stream_of(q))
    _capi.check(code, "decay_scan")
    return out


def decay_table(decays, device) -> torch.Tensor:
    """The `[2, heads]` argument of `decay_scan`: decays and their base-2 logarithms (bounded below: a decay of zero forgets)."""
    d = torch.tensor(decays, dtype=torch.float64)
    return torch.stack([d, torch.log2(d.clamp_min(2.0 ** -100))]).to(device=device, dtype=torch.float32)


def delta_scan(q, k, v, decay, beta, dt_bias, a_log, state, out, group):
    """The gated delta rule with a decay per head and key channel (`rlt_delta_scan`); q and k are made unit vectors here.

    q, k `[rows, kv_heads * dim]`, v, out `[rows, heads * vdim]` (q, k and v slices of rows of one stride), raw decay `[rows, heads * dim]` and
    beta `[rows, heads]`, dt_bias float32 `[heads * dim]`, a_log float32 `[heads]`, state float32 `[slots, heads, dim, vdim]`, updated in
    place.  The tensors hold all rows of a step; the group's sequences are worked on."""
    device = _capi.require_cuda(q, k, v, decay, beta, dt_bias, a_log, state, out, group.cu, group.starts, group.slots)
    if state.dim() != 4 or state.dtype != torch.float32 or not state.is_contiguous():
        raise ValueError("state must be contiguous float32 [slots, heads, dim, vdim]")
    slots, heads, dim, vdim = state.shape
    rows, kv_heads = q.shape[0], q.shape[1] // dim
    if q.shape != (rows, kv_heads * dim) or kv_heads < 1 or heads % kv_heads or k.shape != q.shape or v.shape != (rows, heads * vdim) \
            or out.shape != v.shape or decay.shape != (rows, heads * dim) or beta.shape != (rows, heads):
        raise ValueError("q / k [rows, kv_heads * dim], v / out [rows, heads * vdim], decay [rows, heads * dim], beta [rows, heads]")
    if q.stride(0) != k.stride(0) or k.stride(0) != v.stride(0) or any(t.stride(1) != 1 for t in (q, k, v, decay, beta, out)):
        raise ValueError("q, k and v must be column slices of the same rows")
    if q.dtype not in (torch.float32, torch.bfloat16) or any(t.dtype != q.dtype for t in (k, v, decay, beta, out)):
        raise ValueError("q, k, v, decay, beta and out must share float32 or bfloat16")
    for name, t, n in (("dt_bias", dt_bias, heads * dim), ("a_log", a_log, heads)):
        if t.dtype != torch.float32 or t.shape != (n,) or not t.is_contiguous():
            raise ValueError(f"{name} must be contiguous float32 [{n}]")
    if group.sequences == 0:
        return out
    lib, dtype = _capi.load(), _capi.DTYPE_CODES[q.dtype]
    with torch.cuda.device(device):
        nbytes = lib.rlt_delta_scan_workspace_bytes(group.sequences, group.max_new, rows, heads, dim, vdim, dtype)
        workspace = torch.empty(nbytes, dtype=torch.uint8, device=device)
        code = lib.rlt_delta_scan(
            _capi.ptr(q), _capi.ptr(k), _capi.ptr(v), q.stride(0), _capi.ptr(decay), decay.stride(0), _capi.ptr(beta), beta.stride(0),
            _capi.ptr(dt_bias), _capi.ptr(a_log), _capi.ptr(out), out.stride(0), _capi.ptr(state), slots, _capi.ptr(group.cu),
            _capi.ptr(group.starts), _capi.ptr(group.slots), group.sequences, group.max_new, rows, heads, kv_heads, dim, vdim, dtype,
            _capi.ptr(workspace), nbytes, _capi.stream_of(q))
    _capi.check(code, "delta_scan")
    return out


GATES = {False: 0, True: 1, "sigmoid": 1, "silu": 2}


def gated_norm(y, z, weight, out, parts: int, eps: float, *, gate_behind: bool | str = False):
    """`out = rmsnorm(y * silu(z)) * weight`, or with `gate_behind` `rmsnorm(y) * weight * sigmoid(z)` ("silu": silu(z)); the row normed in
    `parts` equal parts; all `[rows, width]`, any row stride; weight None: ones."""
    device = _capi.require_cuda(y, z, weight, out)
    rows, width = y.shape
    if z.shape != y.shape or out.shape != y.shape or (weight is not None and (weight.shape != (width,) or weight.dtype != torch.float32)) \
            or any(t.stride(1) != 1 for t in (y, z, out)) or y.dtype not in _capi.DTYPE_CODES or z.dtype != y.dtype or out.dtype != y.dtype:
        raise ValueError("y, z and out must be [rows, width] of one dtype with unit inner stride, weight float32 [width]")
    if rows == 0:
        return out
    with torch.cuda.device(device):
        code = _capi.load().rlt_gated_norm(_capi.ptr(y), y.stride(0), _capi.ptr(z), z.stride(0), _capi.ptr(weight), _capi.ptr(out),
                                           out.stride(0), rows, width, parts, float(eps), GATES[gate_behind], _capi.DTYPE_CODES[y.dtype],
                                           _capi.stream_of(y))
    _capi.check(code, "gated_norm")
    return out
