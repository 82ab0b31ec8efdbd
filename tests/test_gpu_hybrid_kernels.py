"""Each kernel of the hybrid decoder alone against the plain float64 functions of plain_hybrid.py."""

from types import SimpleNamespace

import pytest
import torch

import plain_hybrid as plain
import vllm_rlt_b200 as rlt

pytestmark = pytest.mark.gpu
BLOCK = 16
DTYPES = [torch.float32, torch.bfloat16]


def close(got, want, dtype, scale=1.0):
    got, want = got.double().cpu(), want.double()
    tolerance = {torch.float32: 2e-5, torch.bfloat16: 1.2e-2}[dtype] * scale
    assert torch.isfinite(got).all()
    error = (got - want).abs() / (want.abs() + want.pow(2).mean().sqrt())
    assert float(error.max()) < tolerance, float(error.max())


def group_of(portions, starts, slots):
    cu = torch.tensor([0, *torch.tensor(portions).cumsum(0).tolist()], dtype=torch.int32, device="cuda")
    as_int = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    return SimpleNamespace(sequences=len(portions), max_new=max(portions), cu=cu, starts=as_int(starts), slots=as_int(slots))


# ---- attention with score terms ------------------------------------------------------------------
def paged_case(portions, contexts, heads, kv_heads, dim, vdim, dtype, seed, peaks=()):
    """Keys and values scattered over shuffled pages whose unwritten slots hold NaN; `peaks`: (sequence, query row of
    the portion, key position) whose score is made to stand out."""
    g = torch.Generator().manual_seed(seed)
    n = len(contexts)
    width = max(-(-c // BLOCK) for c in contexts) + 1
    pages = torch.randperm(n * width + 3, generator=g)
    key = torch.full((len(pages), BLOCK, kv_heads, dim), float("nan"), dtype=dtype)
    value = torch.full((len(pages), BLOCK, kv_heads, vdim), float("nan"), dtype=dtype)
    tables = torch.full((n, width), -1, dtype=torch.int32)
    q, ks, vs, at = [], [], [], 0
    for s, context in enumerate(contexts):
        k = (torch.randn(context, kv_heads, dim, generator=g)).to(dtype)
        v = torch.randn(context, kv_heads, vdim, generator=g).to(dtype)
        qs = torch.randn(portions[s], heads, dim, generator=g).to(dtype)
        for sequence, row, position in peaks:
            if sequence == s:
                direction = torch.randn(dim, generator=g)
                direction = direction / direction.norm()
                qs[row] = (12 * direction).to(dtype)                          # every head of the row ...
                k[position] = (14 * direction * dim ** 0.5).to(dtype)         # ... finds this key: score about 12 * 14
        count = -(-context // BLOCK)
        tables[s, :count] = pages[at:at + count]
        at += count
        for p in range(context):
            key[tables[s, p // BLOCK], p % BLOCK] = k[p]
            value[tables[s, p // BLOCK], p % BLOCK] = v[p]
        q.append(qs), ks.append(k), vs.append(v)
    return q, ks, vs, key, value, tables


def run_scored(q, key, value, tables, contexts, portions, terms, heads, dim, vdim, pad=0):
    rows = sum(portions)
    wide_q = torch.zeros(rows, heads * dim + pad, dtype=key.dtype, device="cuda")
    wide_q[:, :heads * dim] = torch.cat(q).reshape(rows, -1).cuda()
    wide_out = torch.full((rows, heads * vdim + pad), 7.0, dtype=key.dtype, device="cuda")
    cu = torch.tensor([0, *torch.tensor(portions).cumsum(0).tolist()], dtype=torch.int32, device="cuda")
    attention = rlt.B200PagedAttention()
    attention.scored(wide_q[:, :heads * dim].view(rows, heads, dim), wide_out[:, :heads * vdim].view(rows, heads, vdim), key.cuda(),
                     value.cuda(), tables.cuda(), torch.tensor(contexts, dtype=torch.int32, device="cuda"), cu, max(portions), terms)
    if pad:
        assert bool((wide_out[:, heads * vdim:] == 7.0).all())
    return wide_out[:, :heads * vdim].reshape(rows, heads, vdim)


SHAPES = [(6, 2, 24, 40), (4, 4, 64, 64), (6, 2, 64, 64), (8, 2, 128, 128), (3, 1, 128, 128), (4, 1, 96, 160), (5, 5, 20, 12), (2, 2, 256, 64), (16, 1, 16, 8)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", SHAPES)
@pytest.mark.parametrize("portions,contexts", [([1, 1, 1], [1, 17, 530]), ([2, 16, 5], [2, 33, 300]), ([40, 70, 1], [40, 201, 64]), ([150], [150]), ([300, 17], [500, 17])])
def test_scored_attention(dtype, heads, kv_heads, dim, vdim, portions, contexts):
    terms = rlt.ScoreTerms(0.8 * dim ** -0.5, 0.5, 37, True)
    q, k, v, key, value, tables = paged_case(portions, contexts, heads, kv_heads, dim, vdim, dtype, 3)
    got = run_scored(q, key, value, tables, contexts, portions, terms, heads, dim, vdim, pad=16)
    want = torch.cat([plain.attention(q[s].double(), k[s].double(), v[s].double(), terms.scale, 0.5, 37, True, contexts[s] - portions[s])
                      for s in range(len(portions))])
    close(got, want, dtype, 2.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("coef,every,bias", [(0.0, 1, False), (0.0, 1, True), (0.9, 1, False), (0.25, 64, True)])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(4, 2, 128, 128), (4, 2, 64, 64), (4, 2, 32, 48)])
def test_every_score_term_alone(dtype, coef, every, bias, heads, kv_heads, dim, vdim):
    portions, contexts = [1, 90], [200, 130]
    terms = rlt.ScoreTerms(dim ** -0.5, coef, every, bias)
    q, k, v, key, value, tables = paged_case(portions, contexts, heads, kv_heads, dim, vdim, dtype, 5)
    for s in range(2):      # decoded and prompt rows on their own kernels
        got = run_scored(q[s:s + 1], key, value, tables[s:s + 1], contexts[s:s + 1], portions[s:s + 1], terms, heads, dim, vdim)
        close(got, plain.attention(q[s].double(), k[s].double(), v[s].double(), terms.scale, coef, every, bias, contexts[s] - portions[s]),
              dtype, 2.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(4, 2, 128, 128), (4, 2, 64, 64), (4, 2, 48, 64)])
@pytest.mark.parametrize("position", [0, 1, 15, 16, 255, 256, 511, 512, 639])
def test_one_key_that_stands_out_is_found_wherever_it_lies(dtype, heads, kv_heads, dim, vdim, position):
    """The query's match dominates its softmax at any distance and across page, stage and chunk borders: a row that
    looked anywhere else would be off by whole units."""
    context = 640
    terms = rlt.ScoreTerms(dim ** -0.5, 0.1, 50, True)
    for portion in (1, 40):
        q, k, v, key, value, tables = paged_case([portion], [context], heads, kv_heads, dim, vdim, dtype, 11,
                                                 peaks=[(0, portion - 1, position)])
        got = run_scored(q, key, value, tables, [context], [portion], terms, heads, dim, vdim)
        want = plain.attention(q[0].double(), k[0].double(), v[0].double(), terms.scale, 0.1, 50, True, context - portion)
        close(got, want, dtype, 2.0)
        near = want[-1, -1] - v[0][position, -1].double()      # the last head's slope is the gentlest: it must have landed on the key
        assert float(near.abs().max()) < 0.1


# ---- elementwise kernels -------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,width", [(1, 52), (5, 96), (3, 2048), (2, 33)])
def test_residual_norm(dtype, rows, width):
    g = torch.Generator().manual_seed(rows)
    embed, delta = torch.randn(19, width, generator=g).to(dtype), torch.randn(rows, width, generator=g).to(dtype)
    weight, tokens = torch.randn(width, generator=g), torch.randint(0, 19, (rows,), generator=g)
    residual = torch.full((rows, width), float("nan"), device="cuda")
    out = rlt.residual_norm(residual, weight.cuda(), 1e-3, dtype, tokens=tokens.cuda(), embed=embed.cuda(), weight_offset=1.0)
    x = embed.double()[tokens]
    close(residual, x, torch.float32)
    close(out, plain.norm(x, weight.double(), 1e-3), dtype)
    out = rlt.residual_norm(residual, weight.cuda(), 1e-3, dtype, delta=delta.cuda())
    x = x + delta.double()
    close(residual, x, torch.float32)                          # the sum itself stays in 32 bits
    close(out, plain.norm(x, weight.double(), 1e-3, offset=0.0), dtype)
    rows_wanted = torch.tensor([rows - 1, 0, rows - 1])
    before = residual.clone()
    out = rlt.residual_norm(residual, weight.cuda(), 1e-3, dtype, delta=delta.cuda(), row_index=rows_wanted.cuda(), weight_offset=1.0, store=False)
    assert torch.equal(residual, before)
    close(out, plain.norm(x + delta.double(), weight.double(), 1e-3)[rows_wanted], dtype)


def test_residual_norm_uses_eps_inside_the_root():
    tiny = torch.full((1, 64), 1e-4, device="cuda")
    out = rlt.residual_norm(tiny, torch.zeros(64, device="cuda"), 1e-6, torch.float32, weight_offset=1.0)
    close(out, torch.full((1, 64), 1e-4 / (1e-8 + 1e-6) ** 0.5, dtype=torch.float64), torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kv_heads,dim,vdim,ff,kind", [(2, 24, 40, 72, "gelu"), (1, 5, 3, 9, "gelu_tanh"), (4, 64, 64, 0, None), (0, 0, 0, 40, "gelu")])
def test_block_epilogue(dtype, kv_heads, dim, vdim, ff, kind):
    g = torch.Generator().manual_seed(2)
    k_width, v_width = kv_heads * dim, kv_heads * vdim
    columns = 8 + k_width + v_width + ff
    rows = 6
    proj = (2 * torch.randn(rows, columns, generator=g)).to(dtype).cuda()
    tables = torch.tensor([[4, 1], [0, 5]], dtype=torch.int32, device="cuda")
    row_seq = torch.tensor([0, 0, 1, 1, -1, 1], dtype=torch.int32, device="cuda")
    positions = torch.tensor([15, 16, 0, 31, 3, 32], dtype=torch.int32, device="cuda")     # the last lies behind its table
    batch = SimpleNamespace(tables=tables[None], row_seq=row_seq, positions=positions)
    key = torch.full((6, BLOCK, max(kv_heads, 1), max(dim, 1)), 9.0, dtype=dtype, device="cuda")
    value = torch.full((6, BLOCK, max(kv_heads, 1), max(vdim, 1)), 9.0, dtype=dtype, device="cuda")
    out = torch.full((rows, ff + 8), 9.0, dtype=dtype, device="cuda")
    rlt.block_epilogue(proj, batch, kv=(8, 8 + k_width, key, value) if kv_heads else None,
                       act=(8 + k_width + v_width, ff, kind, out, 8) if ff else None)
    want_key, want_value = torch.full_like(key, 9.0), torch.full_like(value, 9.0)
    if kv_heads:
        for row, (page, slot) in enumerate([(4, 15), (1, 0), (0, 0), (5, 15)]):
            want_key[page, slot] = proj[row, 8:8 + k_width].view(kv_heads, dim)
            want_value[page, slot] = proj[row, 8 + k_width:8 + k_width + v_width].view(kv_heads, vdim)
    assert torch.equal(key, want_key) and torch.equal(value, want_value)
    assert bool((out[:, :8] == 9.0).all())
    if ff:
        x = proj[:, 8 + k_width + v_width:].double().cpu()
        close(out[:, 8:], plain.gelu(x) if kind == "gelu" else plain.gelu_tanh(x), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["gelu", "gelu_tanh"])
def test_activations_over_their_whole_range(dtype, kind):
    x = torch.cat([torch.linspace(-40, 40, 4001), torch.linspace(-1e-3, 1e-3, 95)]).to(dtype).view(8, 512)
    out = torch.empty(8, 512, dtype=dtype, device="cuda")
    rlt.block_epilogue(x.cuda(), None, act=(0, 512, kind, out, 0))
    want = (plain.gelu if kind == "gelu" else plain.gelu_tanh)(x.double())
    error = (out.double().cpu() - want).abs()
    relative = 2.0 ** -8 if dtype == torch.bfloat16 else 4e-6
    assert bool((error <= relative * want.abs() + 2e-6).all())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,parts", [(64, 1), (96, 4), (30, 3), (512, 8)])
def test_gated_norm(dtype, width, parts):
    g = torch.Generator().manual_seed(7)
    y, z = (torch.randn(5, width + 8, generator=g).to(dtype) for _ in range(2))
    y[:, :width // parts] *= 30                                # parts of very different size: each has its own root mean square
    weight = torch.randn(width, generator=g)
    out = torch.full((5, width + 8), 9.0, dtype=dtype, device="cuda")
    rlt.gated_norm(y.cuda()[:, :width], z.cuda()[:, :width], weight.cuda(), out[:, :width], parts, 1e-5)
    close(out[:, :width], plain.gated_norm(y[:, :width].double(), z[:, :width].double(), weight.double(), parts, 1e-5), dtype)
    assert bool((out[:, width:] == 9.0).all())


# ---- recurrent kernels ---------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("channels,taps", [(40, 4), (130, 4), (37, 2), (24, 1), (16, 7)])
@pytest.mark.parametrize("cuts", [[1] * 9, [2, 3, 1, 40, 2], [33, 32, 31], [96]])
def test_convolution_in_portions(dtype, channels, taps, cuts):
    """Two sequences side by side, portion by portion; a freed slot's leftovers must not leak into the next sequence."""
    g = torch.Generator().manual_seed(taps)
    total = sum(cuts)
    x = [torch.randn(total, channels, generator=g).to(dtype) for _ in range(2)]
    weight, bias = torch.randn(channels, taps, generator=g), torch.randn(channels, generator=g)
    state = torch.full((3, taps - 1, channels), 1e4, dtype=dtype, device="cuda")
    slots, got, at = [2, 0], [[], []], 0
    up = torch.randn(2 * total, 24, generator=g).to(dtype)
    for n in cuts:
        rows = torch.cat([s[at:at + n] for s in x])
        wide = torch.cat([rows, up[:2 * n]], 1).cuda()
        out = torch.empty(2 * n, channels, dtype=dtype, device="cuda")
        acted = torch.empty(2 * n, 24, dtype=dtype, device="cuda")
        rlt.causal_conv(wide[:, :channels], weight.cuda(), bias.cuda(), state, out, group_of([n, n], [at, at], slots),
                        act=(wide[:, channels:], "gelu", acted))
        close(acted, plain.gelu(up[:2 * n].double()), dtype)
        for s in range(2):
            got[s].append(out[s * n:(s + 1) * n].cpu())
        at += n
    for s in range(2):
        close(torch.cat(got[s]), plain.convolution(x[s].double(), weight.double(), bias.double()), dtype)
        if taps > 1:
            assert torch.equal(state[slots[s]].cpu(), x[s][total - taps + 1:])
    assert bool((state[1] == 1e4).all())


SCANS = [(4, 16, 20, 2), (3, 10, 12, 3), (2, 64, 128, 1), (2, 32, 48, 2), (2, 80, 144, 1), (1, 7, 9, 1), (2, 64, 256, 2), (4, 24, 64, 4),
         (4, 64, 96, 2), (2, 48, 72, 1), (3, 128, 128, 3)]


def scan_inputs(total, heads, p, size, groups, dtype, seed):
    g = torch.Generator().manual_seed(seed)
    x, b, c = (torch.randn(total, n, generator=g).to(dtype) for n in (heads * p, groups * size, groups * size))
    dt = torch.randn(total, heads, generator=g).to(dtype)
    a_log = torch.linspace(-6.0, 2.0, heads) if heads > 1 else torch.tensor([-4.0])       # memory from thousands of tokens down to one
    return x, b, c, dt, torch.randn(heads, generator=g) - 1, a_log, torch.randn(heads, generator=g)


def run_scan(inputs, cuts, heads, p, size, groups, dtype, state, slots, portions_of):
    x, b, c, dt, dt_bias, a_log, d = inputs
    got, at = [[] for _ in slots], 0
    for n in cuts:
        pick = lambda t: torch.cat([s[at:at + n] for s in portions_of(t)])
        wide = torch.cat([pick(x), pick(b), pick(c)], 1).cuda()
        out = torch.full((wide.shape[0], heads * p), float("nan"), dtype=dtype, device="cuda")
        xs, bs, cs = wide.split((heads * p, groups * size, groups * size), 1)
        rlt.ssd_scan(xs, bs, cs, pick(dt).cuda(), dt_bias.cuda(), a_log.cuda(), d.cuda(), state, out,
                     group_of([n] * len(slots), [at] * len(slots), slots))
        for s in range(len(slots)):
            got[s].append(out[s * n:(s + 1) * n].cpu())
        at += n
    return [torch.cat(g) for g in got]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,p,size,groups", SCANS)
@pytest.mark.parametrize("cuts", [[1] * 6, [2, 16, 17, 64, 3, 65], [167], [129, 127, 20]])
def test_scan_in_portions(dtype, heads, p, size, groups, cuts):
    total = sum(cuts)
    inputs = scan_inputs(2 * total, heads, p, size, groups, dtype, heads * p + size)
    state = torch.full((4, heads, size, p), 1e3, device="cuda")
    halves = lambda t: (t[:total], t[total:])
    got = run_scan(inputs, cuts, heads, p, size, groups, dtype, state, [3, 1], halves)
    x, b, c, dt, dt_bias, a_log, d = (t.double() for t in inputs)
    for s in range(2):
        part = [halves(t)[s] for t in (x, b, c, dt)]
        y, final = plain.recurrence(part[0].view(total, heads, p), part[1].view(total, groups, size), part[2].view(total, groups, size),
                                    part[3], dt_bias, a_log, d)
        close(got[s], y.reshape(total, -1), dtype)
        # inputs are the same 16-bit numbers on both sides: the state itself must be good to far more than 16 bits
        close(state[[3, 1][s]], final, torch.float32, 20.0)
    assert bool((state[0] == 1e3).all()) and bool((state[2] == 1e3).all())


@pytest.mark.parametrize("p,size", [(32, 64), (64, 128), (72, 104)])
def test_long_prompts_run_in_segments(p, size):
    """One long sequence beside a short one: the long one is cut into segments that start from folded states."""
    heads, groups, lengths = 2, 1, [1500, 300]
    inputs = scan_inputs(sum(lengths), heads, p, size, groups, torch.bfloat16, 5)
    x, b, c, dt, dt_bias, a_log, d = inputs
    state = torch.randn(3, heads, size, p, device="cuda")
    start = state.clone()
    wide = torch.cat([x, b, c], 1).cuda()
    out = torch.empty(sum(lengths), heads * p, dtype=torch.bfloat16, device="cuda")
    xs, bs, cs = wide.split((heads * p, size, size), 1)
    rlt.ssd_scan(xs, bs, cs, dt.cuda(), dt_bias.cuda(), a_log.cuda(), d.cuda(), state, out, group_of(lengths, [40, 7], [1, 0]))
    at = 0
    for s, n in enumerate(lengths):
        part = [t[at:at + n].double() for t in (x, b, c, dt)]
        y, final = plain.recurrence(part[0].view(n, heads, p), part[1].view(n, groups, size), part[2].view(n, groups, size), part[3],
                                    dt_bias.double(), a_log.double(), d.double(), start[[1, 0][s]].double().cpu())
        close(out[at:at + n], y.reshape(n, -1), torch.bfloat16)
        close(state[[1, 0][s]], final, torch.float32, 20.0)
        at += n
    assert torch.equal(state[2], start[2])


def test_kernels_refuse_what_they_cannot_do():
    with pytest.raises(ValueError, match="multiple"):
        rlt.B200PagedAttention().scored(torch.zeros(1, 3, 16, device="cuda"), torch.zeros(1, 3, 16, device="cuda"),
                                        torch.zeros(1, 16, 2, 16, device="cuda"), torch.zeros(1, 16, 2, 16, device="cuda"),
                                        torch.zeros(1, 1, dtype=torch.int32, device="cuda"), torch.ones(1, dtype=torch.int32, device="cuda"),
                                        torch.tensor([0, 1], dtype=torch.int32, device="cuda"), 1, rlt.ScoreTerms(1.0))
    with pytest.raises(NotImplementedError, match="taps"):
        x = torch.zeros(1, 8, device="cuda")
        rlt.causal_conv(x, torch.zeros(8, 40, device="cuda"), torch.zeros(8, device="cuda"), torch.zeros(1, 39, 8, device="cuda"),
                        torch.empty_like(x), group_of([1], [0], [0]))
