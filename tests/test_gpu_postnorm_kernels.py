"""Each kernel of the decoder that norms its sublayers' outputs alone against the plain float64 functions of plain_postnorm.py."""

from types import SimpleNamespace

import pytest
import torch

import plain_postnorm as plain
import vllm_rlt_b200 as rlt
from test_gpu_hybrid_kernels import BLOCK, DTYPES, close, group_of, paged_case
from test_gpu_stream_kernels import larger_pages
from vllm_rlt_b200.engine import KeyRanges
from vllm_rlt_b200.talking_mixer import talking_attention

pytestmark = pytest.mark.gpu


def generator(seed):
    return torch.Generator().manual_seed(seed)


# ---- the residual --------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,width,top", [(1, 33, 1), (5, 52, 3), (7, 96, 2), (4, 2048, 4), (2, 5001, 2), (3, 4096, 8)])
@pytest.mark.parametrize("shared", [True, False])
def test_residual_takes_experts_behind_a_norm_and_goes_on_as_it_is(dtype, rows, width, top, shared):
    g = generator(width)
    x, weight, behind = torch.randn(rows, width, generator=g), torch.randn(width, generator=g), torch.randn(width, generator=g)
    y, values = torch.randn(rows, width, generator=g).to(dtype), torch.randn(rows * top, width, generator=g).to(dtype)
    places, shares = torch.randperm(rows * top, generator=g).int().view(rows, top), torch.rand(rows, top, generator=g)
    delta = (shares.double()[:, :, None] * values.double()[places.long()]).sum(1) + (y.double() if shared else 0)
    want = x.double() + plain.rms_norm(delta, 1e-3, behind.double())
    run = lambda residual, w, **kw: rlt.residual_norm(residual, w, 1e-3, dtype, delta=y.cuda() if shared else None, behind=(behind.cuda(), 1.0),
                                                      parts=(values.cuda(), places.cuda(), shares.cuda()), **kw)
    residual = x.cuda()
    h = run(residual, None)
    close(residual, want, torch.float32)
    assert torch.equal(h, residual.to(dtype))
    index = torch.tensor([rows - 1, 0])
    h = run(x.cuda(), weight.cuda(), row_index=index.cuda(), store=False)
    close(h, plain.rms_norm(want, 1e-3, weight.double())[index], dtype)
    residual = x.cuda()
    close(rlt.residual_norm(residual, None, 1e-3, dtype, parts=(values.cuda(), places.cuda(), shares.cuda())),
          x.double() + (shares.double()[:, :, None] * values.double()[places.long()]).sum(1), dtype)       # no norm behind


@pytest.mark.parametrize("dtype", DTYPES)
def test_residual_starts_as_the_embedding(dtype):
    embed, tokens = torch.randn(13, 50, generator=generator(1)).to(dtype), torch.tensor([4, 0, 12, 4])
    residual = torch.full((4, 50), float("nan"), device="cuda")
    h = rlt.residual_norm(residual, None, 1e-3, dtype, tokens=tokens.cuda(), embed=embed.cuda())
    assert torch.equal(residual.cpu(), embed[tokens].float()) and torch.equal(h.cpu(), embed[tokens])


# ---- norms per head with a gate behind ------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim", [(4, 32), (3, 7), (2, 128), (5, 96), (2, 200), (3, 512), (2, 1000), (1, 64), (2, 1)])
@pytest.mark.parametrize("gate", ["sigmoid", "silu", False])
@pytest.mark.parametrize("weighted", [True, False])
def test_norm_per_head_with_a_gate(dtype, heads, dim, gate, weighted):
    g, width = generator(dim), heads * dim
    y, z = ((3 * torch.randn(5, width + 8, generator=g)).to(dtype)[:, :width] for _ in range(2))
    weight = torch.randn(width, generator=g) if weighted else None
    out = torch.full((5, width + 8), 9.0, dtype=dtype, device="cuda")
    rlt.gated_norm(y.cuda(), z.cuda(), None if weight is None else weight.cuda(), out[:, :width], heads, 1e-2, gate_behind=gate)
    a, b = y.double(), z.double()
    if not gate:
        a = a * plain.silu(b)
    want = plain.rms_norm(a.view(5, heads, dim), 1e-2).view(5, width) * (1.0 if weight is None else weight.double())
    if gate:
        want = want * (plain.sigmoid(b) if gate == "sigmoid" else plain.silu(b))
    close(out[:, :width], want, dtype)
    assert bool((out[:, width:] == 9.0).all())


# ---- norm and rotation of queries and keys --------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,dims", [(6, 2, 96, 96, 48), (4, 4, 64, 32, 64), (3, 1, 9, 7, 4), (2, 2, 128, 128, 2), (5, 1, 200, 136, 64),
                                                          (8, 2, 32, 64, 16), (1, 1, 300, 3, 300), (2, 1, 16, 8, 0)])
@pytest.mark.parametrize("halves", [False, True])
@pytest.mark.parametrize("normed", [True, False])
def test_norm_and_rotation_into_pages(dtype, heads, kv_heads, dim, vdim, dims, halves, normed):
    g, starts, counts = generator(dim), [0, 100_000 % 4000, 13], [5, 1, 20]
    rows = sum(counts)
    positions = torch.cat([torch.arange(s, s + n) for s, n in zip(starts, counts)]).int()
    row_seq = torch.cat([torch.full((n,), i) for i, n in enumerate(counts)]).int()
    widths = [heads * dim, kv_heads * dim, kv_heads * vdim]
    columns, at = [], 0
    for n in widths:
        columns.append(at)
        at += -(-n // 8) * 8
    proj = torch.randn(rows, at + 8, generator=g).to(dtype)
    weights = [1 + 0.3 * torch.randn(dim, generator=g) for _ in range(2)] if normed else [None, None]
    pages = max(s + n for s, n in zip(starts, counts)) // BLOCK + 1
    tables = torch.full((1, 3, pages), -1, dtype=torch.int32)
    free = torch.randperm(3 * pages, generator=g)
    for s in range(3):
        for p in range(starts[s] // BLOCK, (starts[s] + counts[s] - 1) // BLOCK + 1):
            tables[0, s, p] = free[s * pages + p]
    key = torch.full((3 * pages, BLOCK, kv_heads, dim), 5.0, dtype=dtype, device="cuda")
    value = torch.full((3 * pages, BLOCK, kv_heads, vdim), 5.0, dtype=dtype, device="cuda")
    row_seq[2] = -1                                                   # a padding row: nothing of it is stored
    batch = SimpleNamespace(row_seq=row_seq.cuda(), positions=positions.cuda(), tables=tables.cuda())
    q = torch.empty(rows, heads, dim, dtype=dtype, device="cuda")
    frequencies = rlt.rotation_frequencies(1e4, dims, "cuda")
    rlt.norm_rotate(proj.cuda(), columns, *(None if w is None else w.cuda() for w in weights), 1e-3, frequencies, q, key, value, batch, halves=halves)
    split = [proj.double()[:, c:c + n].reshape(rows, -1, d) for c, n, d in zip(columns, widths, (dim, dim, vdim))]
    turned = [plain.rotate(plain.rms_norm(x, 1e-3, w.double()) if normed else x, positions, 1e4, dims, halves) for x, w in zip(split, weights)]
    close(q, turned[0], dtype)
    stored = 0
    for r in range(rows):
        if row_seq[r] < 0:
            continue
        page, offset = tables[0, row_seq[r], positions[r] // BLOCK], positions[r] % BLOCK
        close(key[page, offset], turned[1][r], dtype, 2.0)
        assert torch.equal(value[page, offset].cpu().double(), split[2][r])
        stored += 1
    assert int((key != 5.0).any(-1).any(-1).sum()) == int((value != 5.0).any(-1).any(-1).sum()) == stored


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,dims,halves", [(4, 32, 32, True), (3, 7, 2, True), (6, 128, 64, True), (2, 24, 16, False)])
def test_the_last_heads_are_scaled_whole(dtype, heads, dim, dims, halves):
    x, positions = torch.randn(5, heads, dim, generator=generator(3)).to(dtype), torch.tensor([0, 1, 77, 5000, 123456], dtype=torch.int32)
    out = rlt.rotate_heads(x.cuda(), torch.empty_like(x).cuda(), rlt.rotation_frequencies(1e3, dims, "cuda"), positions.cuda(), halves=halves, scale=0.3,
                           scaled_from=heads - 2)
    want = plain.rotate(x.double(), positions, 1e3, dims, halves)
    want[:, heads - 2:] *= 0.3
    close(out, want, dtype)


# ---- bounded scores, kept keys, talking heads ------------------------------------------------------
def talk_of(heads, seed):
    return torch.eye(heads) + 0.5 * torch.randn(heads, heads, generator=generator(seed))


def run_talking(case, contexts, portions, terms, talk, heads, vdim):
    q, _, _, key, value, tables = case
    rows, kv_heads, to = sum(portions), key.shape[2], lambda t: t.cuda()
    cu = torch.tensor([0, *torch.tensor(portions).cumsum(0).tolist()], dtype=torch.int32, device="cuda")
    out = torch.full((rows, heads, vdim), 7.0, dtype=key.dtype, device="cuda")
    group = SimpleNamespace(sequences=len(portions), max_new=max(portions), tables=to(tables), cu=cu, local_cu=cu,
                            lengths=torch.tensor(contexts, dtype=torch.int32, device="cuda"), rows=slice(0, rows),
                            portions=[(c - n, n) for c, n in zip(contexts, portions)])
    group.key_ranges = lambda *which: KeyRanges.of(group.portions, which[0], torch.device("cuda"), *which[1:])
    talking_attention(rlt.B200PagedAttention(), torch.cat(q).cuda(), to(key), to(value), out, group, terms, talk.cuda())
    return out


def plain_talking(case, contexts, portions, terms, talk):
    q, k, v = ([t.double() for t in x] for x in case[:3])
    return torch.cat([plain.talking_attention(q[s], k[s], v[s], terms.scale, terms.head_scale.double().cpu(), terms.softcap, terms.window,
                                              terms.keep_first, talk.double(), contexts[s] - portions[s]) for s in range(len(portions))])


def terms_of(heads, dim, window, keep, cap, seed=1):
    temp = 1 + 0.4 * torch.randn(heads, generator=generator(seed))
    return rlt.ScoreTerms(2.0 * dim ** -0.5, window=window, keep_first=keep, softcap=cap, head_scale=temp.cuda())


SHAPES = [(6, 2, 96, 96), (4, 4, 24, 40), (16, 2, 128, 128), (3, 1, 9, 7), (8, 4, 64, 128), (20, 4, 32, 32), (5, 1, 128, 24), (12, 4, 72, 136), (2, 2, 16, 8),
          (16, 8, 40, 64)]
PORTIONS = [([1, 1, 3], [1, 130, 201]), ([2, 16, 5], [2, 33, 300]), ([1], [900]), ([70, 150, 17], [70, 230, 500]), ([300, 40], [300, 41])]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", SHAPES)
@pytest.mark.parametrize("window,keep,cap,page", [(40, 4, 15.0, 16), (40, 0, 3.0, 64), (1, 1, 15.0, 64), (64, 70, 40.0, 64), (130, 65, 90.0, 16), (1000, 8, 15.0, 64)])
def test_talking_attention(dtype, heads, kv_heads, dim, vdim, window, keep, cap, page):
    terms, talk = terms_of(heads, dim, window, keep, cap), talk_of(heads, 2)
    for portions, contexts in PORTIONS:
        case = paged_case(portions, contexts, heads, kv_heads, dim, vdim, dtype, 4)
        want = plain_talking(case, contexts, portions, terms, talk)
        if page > BLOCK:
            key, tables = larger_pages(case[3], case[5], page)
            value, _ = larger_pages(case[4], case[5], page)
            case = (*case[:3], key, value, tables)
        close(run_talking(case, contexts, portions, terms, talk, heads, vdim), want, dtype, 3 * float(talk.norm(dim=1).max()))    # mixing adds up roundings


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(6, 2, 96, 96), (16, 2, 128, 128), (3, 1, 9, 7)])
@pytest.mark.parametrize("window,keep", [(40, 5), (64, 1), (17, 64), (65, 70)])
def test_keys_at_the_edges_of_window_and_kept_tokens(dtype, heads, kv_heads, dim, vdim, window, keep):
    """One key stands out for the last row of the portion: the answer shows it just inside an edge, and does not know it just outside."""
    terms, talk = terms_of(heads, dim, window, keep, 30.0), torch.eye(heads)
    for n, context in ((1, 200), (3, 200), (90, 200), (200, 200)):
        row = n - 1
        for position in (0, keep - 1, keep, context - window - 1, context - window, context - 1, 15, 16, 63, 64):
            case = paged_case([n], [context], heads, kv_heads, dim, vdim, dtype, 6, peaks=[(0, row, position)])
            got = run_talking(case, [context], [n], terms, talk, heads, vdim)
            close(got, plain_talking(case, [context], [n], terms, talk), dtype, 2.5)
            case[2][0][position] += 50.0                              # another value under the same key
            page = case[5][0, position // BLOCK]
            case[4][page, position % BLOCK] += 50.0
            moved = (run_talking(case, [context], [n], terms, talk, heads, vdim) - got).abs()[-1].max() > 0
            assert bool(moved) == (position < keep or context - 1 - position < window), (n, position)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,heads,kv_heads,dim", [(1, 1, 1, 5), (3, 6, 2, 96), (5, 16, 4, 128), (2, 33, 3, 24), (2, 96, 96, 8)])
def test_heads_are_mixed_behind_the_softmax(dtype, rows, heads, kv_heads, dim):
    g = generator(rows)
    y, talk = torch.randn(rows, heads, kv_heads * dim, generator=g).to(dtype), torch.randn(heads, heads, generator=g)
    out = rlt.head_mix(y.cuda(), talk.cuda(), torch.empty(rows, heads, dim, dtype=dtype, device="cuda"), kv_heads)
    spread = y.double().view(rows, heads, kv_heads, dim)
    own = torch.arange(heads) // (heads // kv_heads)
    want = torch.stack([torch.einsum("g,ngd->nd", talk[h].double(), spread[:, :, own[h]]) for h in range(heads)], 1)
    close(out, want, dtype, 2.0)


# ---- the gated delta rule ---------------------------------------------------------------------------
def delta_case(total, heads, kv_heads, dim, vdim, dtype, seed, strong=False, repeat=False):
    """Rows [q | k | v | decay | beta] as the projections leave them; `strong`: decays down to exp(-30) a token; `repeat`: equal keys and
    hardly any decay, where a read before the write matters most."""
    g = generator(seed)
    sizes = [kv_heads * dim, kv_heads * dim, heads * vdim, heads * dim, heads]
    parts = [torch.randn(total, n, generator=g) for n in sizes]
    if repeat:
        parts[1] = parts[1][:1] + 0.05 * parts[1]
        parts[4] = 2 + parts[4]
    a_log, dt_bias = torch.linspace(-2.0, 1.0, heads), -3.0 + 1.5 * torch.randn(heads * dim, generator=g)
    if strong:
        a_log, dt_bias = torch.linspace(0.0, 3.0, heads), torch.randn(heads * dim, generator=g)
    if repeat:
        dt_bias = dt_bias - 6
    return [p.to(dtype) for p in parts], a_log, dt_bias


def plain_delta(parts, a_log, dt_bias, heads, kv_heads, dim, vdim, state=None):
    q, k, v, decay, beta = (p.double() for p in parts)
    n, own = q.shape[0], torch.arange(heads) // (heads // kv_heads)
    q, k = (plain.unit_vector(x.view(n, kv_heads, dim))[:, own] for x in (q, k))
    log_decay = plain.channel_decay(decay.view(n, heads, dim), a_log.double(), dt_bias.double().view(heads, dim))
    return plain.delta_rule(q * dim ** -0.5, k, v.view(n, heads, vdim), log_decay, plain.sigmoid(beta), state)


def feed_delta(cases, a_log, dt_bias, cuts, heads, kv_heads, dim, vdim, dtype):
    """All sequences in portions of `cuts` side by side; outputs per sequence, and the slots."""
    state = torch.full((len(cases) + 2, heads, dim, vdim), float("nan"), device="cuda")
    slots, got, at = [len(cases) - s for s in range(len(cases))], [[] for _ in cases], 0
    pad = lambda x: torch.cat([x, torch.zeros(x.shape[0], -x.shape[1] % 8, dtype=x.dtype)], 1)
    for n in cuts:
        rows = [torch.cat([c[i][at:at + n] for c in cases]) for i in range(5)]
        offsets, total, wide = [], 0, []
        for r in rows[:3]:
            offsets.append(total)
            wide.append(pad(r))
            total += wide[-1].shape[1]
        qkv = torch.cat(wide, 1).cuda()
        q, k, v = (qkv[:, o:o + r.shape[1]] for o, r in zip(offsets, rows[:3]))
        out = torch.empty(n * len(cases), heads * vdim, dtype=dtype, device="cuda")
        rlt.delta_scan(q, k, v, rows[3].cuda(), pad(rows[4]).cuda()[:, :heads], dt_bias.cuda(), a_log.cuda(), state, out,
                       group_of([n] * len(cases), [at] * len(cases), slots))
        for s in range(len(cases)):
            got[s].append(out[s * n:(s + 1) * n].view(n, heads, vdim))
        at += n
    return [torch.cat(g) for g in got], state, slots


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(4, 4, 32, 32), (4, 2, 128, 128), (3, 1, 9, 7), (2, 2, 64, 72), (2, 1, 80, 200), (1, 1, 200, 16), (2, 2, 24, 130)])
@pytest.mark.parametrize("cuts", [[150], [64, 65, 21], [1, 2, 16, 17, 63, 51], [130, 1, 1, 18], [40, 110]], ids=str)
def test_delta_rule_in_portions(dtype, heads, kv_heads, dim, vdim, cuts):
    cases = [delta_case(sum(cuts), heads, kv_heads, dim, vdim, dtype, seed)[0] for seed in (1, 2)]
    _, a_log, dt_bias = delta_case(1, heads, kv_heads, dim, vdim, dtype, 1)
    got, state, slots = feed_delta(cases, a_log, dt_bias, cuts, heads, kv_heads, dim, vdim, dtype)
    for s, case in enumerate(cases):
        want, last = plain_delta(case, a_log, dt_bias, heads, kv_heads, dim, vdim)
        close(got[s], want, dtype)
        close(state[slots[s]], last, torch.float32, 3.0)
    assert bool(state[0].isnan().all() and state[3].isnan().all())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["strong", "repeat"])
@pytest.mark.parametrize("dim,vdim", [(128, 128), (48, 64)])
@pytest.mark.parametrize("cuts", [[200], [100, 64, 30, 6]], ids=str)
def test_delta_rule_with_strong_decays_and_with_equal_keys(dtype, kind, dim, vdim, cuts):
    case, a_log, dt_bias = delta_case(200, 3, 3, dim, vdim, dtype, 5, **{kind: True})
    got, state, slots = feed_delta([case], a_log, dt_bias, cuts, 3, 3, dim, vdim, dtype)
    want, last = plain_delta(case, a_log, dt_bias, 3, 3, dim, vdim)
    close(got[0], want, dtype, 1.5)
    close(state[slots[0]], last, torch.float32, 20.0 if dtype == torch.bfloat16 else 5.0)


@pytest.mark.parametrize("dtype", DTYPES)
def test_delta_rule_of_unequal_portions(dtype):
    """Sequences of different lengths and starts in one call, one of them far longer than the others."""
    heads, kv_heads, dim, vdim, lengths = 2, 1, 64, 64, [700, 3, 65, 17]
    a_log, dt_bias = delta_case(1, heads, kv_heads, dim, vdim, dtype, 1)[1:]
    cases = [delta_case(n, heads, kv_heads, dim, vdim, dtype, 10 + n)[0] for n in lengths]
    before = torch.randn(6, heads, dim, vdim, generator=generator(3))
    state, slots, starts = before.cuda(), [3, 0, 5, 1], [0, 9, 0, 40]
    rows = [torch.cat([c[i] for c in cases]).cuda() for i in range(5)]
    qkv = torch.cat(rows[:3], 1)
    out = torch.empty(sum(lengths), heads * vdim, dtype=dtype, device="cuda")
    q, k, v = qkv.split((kv_heads * dim, kv_heads * dim, heads * vdim), 1)
    rlt.delta_scan(q, k, v, rows[3], rows[4], dt_bias.cuda(), a_log.cuda(), state, out, group_of(lengths, starts, slots))
    at = 0
    for n, start, slot, case in zip(lengths, starts, slots, cases):
        want, last = plain_delta(case, a_log, dt_bias, heads, kv_heads, dim, vdim, before[slot].double() if start else None)
        close(out[at:at + n].view(n, heads, vdim), want, dtype)
        close(state[slot], last, torch.float32, 3.0)
        at += n
    assert torch.equal(state[2].cpu(), before[2]) and torch.equal(state[4].cpu(), before[4])


# ---- experts ----------------------------------------------------------------------------------------
@pytest.mark.parametrize("rows,experts,top", [(1, 4, 1), (17, 16, 4), (300, 60, 6), (5000, 9, 9), (40, 200, 3)])
def test_routing_by_biased_logits(rows, experts, top):
    g = generator(experts)
    logits, bias = 3 * torch.randn(rows, experts, generator=g), 2 * torch.randn(experts, generator=g)
    routing = rlt.expert_route(logits.cuda(), None, top, bias=bias.cuda(), floor_sum=0.0)
    z = (logits + bias).double()
    best, order = z.topk(top, dim=1)
    assert torch.equal(routing.chosen.cpu().long().sort(1).values, order.sort(1).values)
    assert torch.allclose(routing.weights.cpu().double(), torch.softmax(best, 1), atol=1e-6)
    assert torch.equal(routing.counts.cpu().long(), torch.bincount(order.flatten(), minlength=experts))


def test_routing_of_logits_far_apart():
    """Scores that underflow are still told apart by their logits."""
    logits = torch.tensor([[0.0, -300.0, 200.0, -200.0, -250.0]])
    routing = rlt.expert_route(logits.cuda(), None, 3, floor_sum=0.0)
    assert sorted(routing.chosen[0].tolist()) == [0, 2, 3] and float(routing.weights.sum()) == pytest.approx(1.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("inner,ff,counts", [(96, 40, [3, 0, 17, 1]), (52, 11, [5, 2]), (256, 96, [40, 130, 7, 0, 300]), (64, 200, [1000, 20]), (24, 4, [1])])
def test_paired_expert_products(dtype, inner, ff, counts):
    g = generator(ff)
    x = torch.randn(sum(counts), inner, generator=g).to(dtype)
    gate, up = ((torch.randn(len(counts), ff, inner, generator=g) / inner ** 0.5).to(dtype) for _ in range(2))
    paired = rlt.paired_rows(gate, up)
    assert torch.equal(paired[:, 0::2], gate) and torch.equal(paired[:, 1::2], up)
    got = rlt.expert_gemm(x.cuda(), paired.cuda(), torch.tensor(counts, dtype=torch.int32, device="cuda"), "silu", paired=True)
    own = torch.repeat_interleave(torch.arange(len(counts)), torch.tensor(counts))
    a, b = (torch.einsum("ni,nfi->nf", x.double(), w.double()[own]) for w in (gate, up))
    assert got.shape == (sum(counts), ff)
    close(got, plain.silu(a) * b, dtype)
