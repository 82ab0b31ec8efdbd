"""Each kernel of the decoder over hyper-connected streams alone against the plain float64 functions of plain_stream.py."""

from types import SimpleNamespace

import pytest
import torch

import plain_hybrid
import plain_stream as plain
import vllm_rlt_b200 as rlt
from test_gpu_hybrid_kernels import BLOCK, DTYPES, close, group_of, paged_case, run_scored
from vllm_rlt_b200.engine import KeyRanges

pytestmark = pytest.mark.gpu


# ---- streams -------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,count,width", [(1, 1, 52), (5, 2, 96), (3, 4, 2048), (4, 3, 33), (2, 8, 64), (3, 5, 40)])
def test_streams_between_two_sublayers(dtype, rows, count, width):
    g = torch.Generator().manual_seed(rows * count)
    f = lambda *shape: torch.randn(*shape, generator=g)
    streams, delta, weight = f(rows, count, width), f(rows, width).to(dtype), f(width)
    out, mix, reads = f(count), f(count, count), f(count)                       # mix is not symmetric: from and to must not be swapped
    gpu = streams.cuda()
    h = rlt.stream_mix(gpu, weight.cuda(), 1e-3, dtype, delta=delta.cuda(), ran=(out.cuda(), mix.cuda()), follows=reads.cuda())
    want = plain.write_streams(list(streams.double().unbind(1)), delta.double(), out.double(), mix.double())
    close(gpu, torch.stack(want, 1), torch.float32)                             # the streams stay in 32 bits
    close(h, plain.rms_norm(plain.read_streams(want, reads.double()), weight.double(), 1e-3), dtype)
    # selected rows, the plain sum, nothing stored
    before, picked = gpu.clone(), torch.tensor([rows - 1, 0, rows - 1])
    h = rlt.stream_mix(gpu, weight.cuda(), 1e-3, dtype, delta=delta.cuda(), ran=(out.cuda(), mix.cuda()), row_index=picked.cuda(), store=False,
                       weight_offset=1.0)
    assert torch.equal(gpu, before)
    want = plain.write_streams(want, delta.double(), out.double(), mix.double())
    close(h, plain.rms_norm(sum(want), 1 + weight.double(), 1e-3)[picked], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("top", [1, 3, 8])
def test_streams_take_weighted_parts(dtype, top):
    g = torch.Generator().manual_seed(top)
    rows, count, width = 7, 2, 72
    streams, delta = torch.randn(rows, count, width, generator=g), torch.randn(rows * top, width, generator=g).to(dtype)
    places = torch.randperm(rows * top, generator=g).view(rows, top).int()
    weights, out, mix = torch.rand(rows, top, generator=g), torch.randn(count, generator=g), torch.randn(count, count, generator=g)
    gpu = streams.cuda()
    rlt.stream_mix(gpu, torch.ones(width, device="cuda"), 1e-5, dtype, delta=delta.cuda(), parts=(places.cuda(), weights.cuda()),
                   ran=(out.cuda(), mix.cuda()))
    y = (delta.double()[places.long()] * weights.double()[:, :, None]).sum(1)
    close(gpu, torch.stack(plain.write_streams(list(streams.double().unbind(1)), y, out.double(), mix.double()), 1), torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("bigram", [None, (11, 5, 3), (1, 0, 1), (4093, 100003, 99991)])
@pytest.mark.parametrize("width", [33, 96])
def test_streams_start_from_the_embedding(dtype, bigram, width):
    g = torch.Generator().manual_seed(4)
    vocab, tokens = 50021, [50020, 3, 50020, 50019, 0, 7]
    embed = torch.randn(vocab, width, generator=g).to(dtype)
    table = torch.randn(bigram[0] + 1, width, generator=g).to(dtype) if bigram else None
    norm, weight, reads = torch.randn(width, generator=g), torch.randn(width, generator=g), torch.tensor([0.3, -1.2, 2.0])
    previous = torch.tensor([-1, *tokens[:-1]], dtype=torch.int32)
    streams = torch.full((6, 3, width), float("nan"), device="cuda")
    h = rlt.stream_mix(streams, weight.cuda(), 1e-2, dtype, follows=reads.cuda(), tokens=torch.tensor(tokens).cuda(), previous=previous.cuda(),
                       embed=embed.cuda(), bigram=(table.cuda(), *bigram[1:]) if bigram else None, embed_weight=norm.cuda())
    x = embed.double()[tokens]
    if bigram:
        x = x + table.double()[plain.bigram_rows(tokens, *bigram)]
    x = plain.rms_norm(x, norm.double(), 1e-2)
    close(streams, x[:, None].expand(6, 3, width), torch.float32)
    close(h, plain.rms_norm(x * reads.double().sum(), weight.double(), 1e-2), dtype)


# ---- latent rows ---------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("q_rank,kv_rank,rot_dim,dims", [(56, 48, 16, 16), (13, 11, 6, 6), (1536, 512, 64, 64), (8, 24, 12, 8), (24, 40, 5, 4)])
def test_latent_rows_are_normed_rotated_and_written(dtype, q_rank, kv_rank, rot_dim, dims):
    g = torch.Generator().manual_seed(3)
    rows, row = 6, kv_rank + rot_dim
    proj = (3 * torch.randn(rows, q_rank + 8 + row, generator=g)).to(dtype)
    wq, wk = torch.randn(q_rank, generator=g), torch.randn(kv_rank, generator=g)
    tables = torch.tensor([[4, 1], [0, 5]], dtype=torch.int32, device="cuda")
    positions = torch.tensor([15, 16, 0, 31, 3, 32], dtype=torch.int32)
    batch = SimpleNamespace(tables=tables[None], row_seq=torch.tensor([0, 0, 1, 1, -1, 1], dtype=torch.int32, device="cuda"), positions=positions.cuda())
    cache = torch.full((6, BLOCK, 1, row), 9.0, dtype=dtype, device="cuda")
    q = rlt.latent_write(proj.cuda(), 0, q_rank + 8, wq.cuda(), wk.cuda(), 1e-3, rlt.rotation_frequencies(70.0, dims, "cuda"), cache, batch)
    close(q, plain.rms_norm(proj[:, :q_rank].double(), wq.double(), 1e-3), dtype)
    down = proj[:, q_rank + 8:].double()
    c = plain.rms_norm(down[:, :kv_rank], wk.double(), 1e-3)
    r = plain.rotate(down[:, kv_rank:], positions, 70.0, dims)
    for i, (page, slot) in enumerate([(4, 15), (1, 0), (0, 0), (5, 15)]):
        close(cache[page, slot, 0, :kv_rank], c[i], dtype)
        close(cache[page, slot, 0, kv_rank:], r[i], dtype)
        cache[page, slot] = 9.0
    assert bool((cache == 9.0).all())             # neither the padding row nor the one behind its table was written


@pytest.mark.parametrize("dtype", DTYPES)
def test_rotation_of_heads_far_into_a_sequence(dtype):
    g = torch.Generator().manual_seed(5)
    q = torch.randn(7, 3, 40, generator=g).to(dtype)
    positions = torch.tensor([0, 1, 63, 1000, 65537, 1 << 20, 123456789], dtype=torch.int32)
    frequencies = rlt.rotation_frequencies(5e4, 16, "cuda")
    want = q.double()
    want[:, :, 24:] = plain.rotate(want[:, :, 24:], positions, 5e4, 16)
    gpu = q.cuda()
    other = torch.zeros(7, 3, 16, dtype=dtype, device="cuda")
    rlt.rotate_heads(gpu[:, :, 24:], other, frequencies, positions.cuda())
    assert torch.equal(gpu.cpu(), q)
    rlt.rotate_heads(gpu[:, :, 24:], gpu[:, :, 24:], frequencies, positions.cuda())
    close(gpu, want, dtype)
    assert torch.equal(other, gpu[:, :, 24:])
    wide = torch.randn(7, 2, 11, generator=g).to(dtype).cuda()                # the dimensions behind the turned ones pass
    turned = rlt.rotate_heads(wide, torch.empty_like(wide), rlt.rotation_frequencies(10.0, 6, "cuda"), positions.cuda())
    assert torch.equal(turned[:, :, 6:], wide[:, :, 6:]) and torch.equal(turned[0], wide[0])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [96, 17])
def test_gathered_rows_are_those_of_the_range(dtype, width):
    g = torch.Generator().manual_seed(6)
    cache = torch.randn(9, BLOCK, 1, width, generator=g).to(dtype).cuda()
    tables = torch.tensor([[3, 0, 7], [8, 2, -1], [5, -1, -1]], dtype=torch.int32, device="cuda")
    portions = [(20, 25), (0, 30), (15, 1)]
    for window in (0, 1, 9, 100):
        ranges = KeyRanges.of(portions, window, cache.device)
        got = rlt.latent_gather(cache, tables, ranges)
        want = [cache[tables[s, p // BLOCK], p % BLOCK, 0] for s, (start, n) in enumerate(portions)
                for p in range(max(start - window + 1, 0) if window else 0, start + n)]
        assert torch.equal(got, torch.stack(want))


# ---- attention with windows ----------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(4, 2, 24, 40), (8, 2, 128, 128), (4, 4, 64, 64), (3, 1, 9, 7)])
@pytest.mark.parametrize("window", [1, 2, 16, 63, 64, 65, 300])
def test_scored_attention_with_a_window(dtype, heads, kv_heads, dim, vdim, window):
    for portions, contexts in (([1, 1, 3], [1, 130, 201]), ([70, 150], [70, 230])):
        q, k, v, key, value, tables = paged_case(portions, contexts, heads, kv_heads, dim, vdim, dtype, window)
        got = run_scored(q, key, value, tables, contexts, portions, rlt.ScoreTerms(dim ** -0.5, window=window), heads, dim, vdim)
        share = heads // kv_heads
        want = torch.cat([plain.windowed_attention(q[s].double(), k[s].double().repeat_interleave(share, 1), v[s].double().repeat_interleave(share, 1),
                                                   dim ** -0.5, window, contexts[s] - portions[s]) for s in range(len(portions))])
        close(got, want, dtype, 2.0)


def latent_case(portions, contexts, heads, row, dtype, seed, peak=None):
    """Cache rows over shuffled pages whose unwritten slots hold NaN.  peak = (distance, strength): the last query row of every
    sequence finds the key that far back."""
    q, k, _, key, _, tables = paged_case(portions, contexts, heads, 1, row, 8, dtype, seed)
    if peak is not None:
        for s, context in enumerate(contexts):
            position = context - 1 - peak[0]
            if position >= 0:
                direction = torch.randn(row, generator=torch.Generator().manual_seed(seed + s))
                direction /= direction.norm()
                q[s][-1] = (peak[1] * direction).to(dtype)
                k[s][position, 0] = (peak[1] * row ** 0.5 * direction).to(dtype)
                key[tables[s, position // BLOCK], position % BLOCK, 0] = k[s][position, 0]
    return q, [x[:, 0] for x in k], key, tables


def run_latent(q, key, tables, contexts, portions, rank, terms):
    rows, heads = sum(portions), q[0].shape[1]
    out = torch.full((rows, heads, rank), 7.0, dtype=key.dtype, device="cuda")
    cu = torch.tensor([0, *torch.tensor(portions).cumsum(0).tolist()], dtype=torch.int32, device="cuda")
    pages = key.cuda()
    rlt.B200PagedAttention().scored(torch.cat(q).cuda(), out, pages, pages[..., :rank], tables.cuda(),
                                    torch.tensor(contexts, dtype=torch.int32, device="cuda"), cu, max(portions), terms)
    return out


def larger_pages(key, tables, size):
    """The same rows over pages of `size` tokens (in an order of their own), unwritten slots NaN."""
    n, width = tables.shape
    per = size // BLOCK
    order = torch.randperm(n * -(-width // per), generator=torch.Generator().manual_seed(size)).view(n, -1)
    pages = torch.full((order.numel(), size, *key.shape[2:]), float("nan"), dtype=key.dtype)
    for s in range(n):
        for i, page in enumerate(tables[s].tolist()):
            if page >= 0:
                pages[order[s, i // per], i % per * BLOCK:(i % per + 1) * BLOCK] = key[page]
    return pages, order.int()


LATENTS = [(6, 48, 16), (16, 512, 64), (20, 72, 24), (1, 4, 2), (5, 11, 6), (32, 256, 32), (40, 128, 64), (3, 64, 8)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,rank,rot", LATENTS)
@pytest.mark.parametrize("window", [0, 1, 40, 64, 129])
@pytest.mark.parametrize("page", [16, 64])
def test_attention_over_cache_rows(dtype, heads, rank, rot, window, page):
    """Every head scores one row per key, and the row's first part is its value: decoded tokens and short portions."""
    row = rank + rot
    terms = rlt.ScoreTerms(0.7 * row ** -0.5, window=window)
    for portions, contexts in (([1, 1, 1], [1, 17, 530]), ([2, 16, 5], [2, 33, 300]), ([1] * 5, [64, 65, 128, 129, 40])):
        q, k, key, tables = latent_case(portions, contexts, heads, row, dtype, 7)
        if page > BLOCK:
            key, tables = larger_pages(key, tables, page)
        got = run_latent(q, key, tables, contexts, portions, rank, terms)
        want = torch.cat([plain.windowed_attention(q[s].double(), k[s].double()[:, None].expand(-1, heads, -1), k[s].double()[:, None, :rank].expand(-1, heads, -1),
                                                   terms.scale, window, contexts[s] - portions[s]) for s in range(len(portions))])
        close(got, want, dtype, 2.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,rank,rot", [(6, 48, 16), (16, 512, 64), (3, 11, 6)])
@pytest.mark.parametrize("window", [16, 50, 64, 300])
def test_a_key_just_inside_a_window_is_found_and_one_just_outside_is_not(dtype, heads, rank, rot, window):
    row, contexts = rank + rot, [420, 333, 301]
    terms = rlt.ScoreTerms(row ** -0.5, window=window)
    for portions in ([1, 1, 1], [2, 9, 16]):
        for distance in (window - 1, window):
            q, k, key, tables = latent_case(portions, contexts, heads, row, dtype, 11, peak=(distance, 12.0))
            if portions[0] == 1:
                key, tables = larger_pages(key, tables, 64)
            got = run_latent(q, key, tables, contexts, portions, rank, terms).double().cpu()
            at = 0
            for s, n in enumerate(portions):
                at += n
                value = k[s][contexts[s] - 1 - distance, :rank].double()
                missed = float((got[at - 1, 0] - value).norm() / value.norm())
                assert missed < 0.05 if distance < window else missed > 0.5


PROMPTS = [([300], [300]), ([17, 64, 129], [17, 200, 129]), ([256, 257, 128], [300, 900, 128]), ([70], [700]), ([40, 600], [41, 600])]


def expanded_case(portions, contexts, heads, dim, rot, vdim, window, seed, peak=None):
    """Packed keys and values of what the portions see.  peak = distance: the last row of every portion finds the key that far back."""
    g = torch.Generator().manual_seed(seed)
    ranges = KeyRanges.of([(c - n, n) for c, n in zip(contexts, portions)], window, torch.device("cuda"))
    q = [torch.randn(n, heads, dim + rot, generator=g).bfloat16() for n in portions]
    k = [torch.randn(c, heads, dim, generator=g).bfloat16() for c in contexts]
    r = [torch.randn(c, rot, generator=g).bfloat16() for c in contexts]
    v = [torch.randn(c, heads, vdim, generator=g).bfloat16() for c in contexts]
    if peak is not None:
        for s, c in enumerate(contexts):
            if c - 1 - peak >= 0:
                direction = torch.randn(dim, generator=g)
                direction /= direction.norm()
                q[s][-1, :, :dim] = (12 * direction).bfloat16()
                k[s][c - 1 - peak] = (12 * (dim + rot) ** 0.5 * direction).bfloat16()
    first = ranges.first.tolist()
    kv = torch.cat([torch.cat([k[s][first[s]:].flatten(1), v[s][first[s]:].flatten(1)], 1) for s in range(len(contexts))])
    shared = torch.cat([torch.cat([torch.full((contexts[s] - first[s], 8), float("nan")).bfloat16(), r[s][first[s]:]], 1) for s in range(len(contexts))])
    out = torch.full((sum(portions), heads, vdim), 7.0, dtype=torch.bfloat16, device="cuda")
    rlt.latent_prompt_attention(torch.cat(q).cuda(), kv.cuda(), shared.cuda()[:, 8:], out, dim, ranges, (dim + rot) ** -0.5, window)
    return q, [torch.cat([k[s], r[s][:, None].expand(-1, heads, -1)], -1) for s in range(len(contexts))], v, out


@pytest.mark.parametrize("heads,dim,rot,vdim", [(3, 128, 64, 128), (2, 64, 32, 80), (5, 40, 8, 64), (2, 72, 64, 24), (1, 8, 16, 128)])
@pytest.mark.parametrize("window", [0, 1, 40, 64, 127, 128, 129, 300])
@pytest.mark.parametrize("portions,contexts", PROMPTS, ids=str)
def test_prompt_attention_over_expanded_latents(heads, dim, rot, vdim, window, portions, contexts):
    assert rlt.latent_prompt_supported(dim, rot, vdim, torch.bfloat16)
    q, k, v, got = expanded_case(portions, contexts, heads, dim, rot, vdim, window, 3)
    want = torch.cat([plain.windowed_attention(q[s].double(), k[s].double(), v[s].double(), (dim + rot) ** -0.5, window, contexts[s] - portions[s])
                      for s in range(len(portions))])
    close(got, want, torch.bfloat16, 2.0)


@pytest.mark.parametrize("heads,dim,rot,vdim", [(2, 128, 64, 128), (2, 64, 32, 80)])
@pytest.mark.parametrize("window", [16, 64, 130, 200])
def test_prompt_rows_find_a_key_just_inside_the_window_and_none_outside(heads, dim, rot, vdim, window):
    portions, contexts = [20, 150, 257, 129], [320, 333, 300, 400]
    for distance in (window - 1, window):
        _, _, v, got = expanded_case(portions, contexts, heads, dim, rot, vdim, window, 5, peak=distance)
        at = 0
        for s, n in enumerate(portions):
            at += n
            value = v[s][contexts[s] - 1 - distance].double()
            missed = float((got[at - 1].double().cpu() - value).norm() / value.norm())
            assert missed < 0.05 if distance < window else missed > 0.5


def test_other_head_sizes_are_left_to_the_general_kernels():
    assert not rlt.latent_prompt_supported(128, 64, 128, torch.float32)
    assert not any(rlt.latent_prompt_supported(*sizes, torch.bfloat16) for sizes in ((136, 64, 128), (128, 72, 128), (128, 64, 136), (60, 32, 64), (64, 30, 64)))


# ---- linear attention ----------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim", [(5, 24, 40), (3, 10, 7), (2, 128, 128), (2, 96, 64), (3, 64, 32), (1, 160, 80)])
@pytest.mark.parametrize("cuts", [[1] * 9, [2, 3, 1, 40, 2], [130, 17, 64], [700]], ids=str)
def test_decayed_attention_in_portions(dtype, heads, dim, vdim, cuts):
    """Two sequences side by side whose slots hold garbage before they start."""
    g = torch.Generator().manual_seed(dim)
    decay = torch.linspace(1.0, 0.4, heads)
    total = sum(cuts)
    x = [(torch.randn(total, heads * (2 * dim + vdim) + 8, generator=g) * 0.4).to(dtype) for _ in range(2)]
    table = rlt.decay_table(decay.tolist(), "cuda")
    state = torch.full((4, heads, dim, vdim), float("nan"), device="cuda")
    slots, got, at = [2, 0], [[], []], 0
    for n in cuts:
        rows = torch.cat([t[at:at + n] for t in x]).cuda()
        q, k, v = rows[:, :heads * dim], rows[:, heads * dim:2 * heads * dim], rows[:, 2 * heads * dim:2 * heads * dim + heads * vdim]
        out = torch.empty(2 * n, heads * vdim, dtype=dtype, device="cuda")
        rlt.decay_scan(q, k, v, table, state, out, group_of([n, n], [at, at], slots))
        for s in range(2):
            got[s].append(out[s * n:(s + 1) * n].view(n, heads, vdim))
        at += n
    for s in range(2):
        split = x[s].double()[:, :heads * (2 * dim + vdim)].split((heads * dim, heads * dim, heads * vdim), 1)
        q, k, v = (t.reshape(total, heads, -1) for t in split)
        want, last = plain.decayed_attention(q, k, v, decay.double())
        close(torch.cat(got[s]), want, dtype)
        close(state[slots[s]], last, torch.float32, 20.0 if dtype == torch.bfloat16 else 2.0)
    assert bool(state[1].isnan().all() and state[3].isnan().all())


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_decay_of_zero_remembers_nothing(dtype):
    g = torch.Generator().manual_seed(9)
    for n in (3, 200):
        rows = torch.randn(n, 3 * 64, generator=g).to(dtype).cuda()
        out, state = torch.empty(n, 64, dtype=dtype, device="cuda"), torch.zeros(1, 2, 32, 32, device="cuda")
        rlt.decay_scan(rows[:, :64], rows[:, 64:128], rows[:, 128:], rlt.decay_table([0.0, 1.0], "cuda"), state, out, group_of([n], [0], [0]))
        q, k, v = (t.reshape(n, 2, 32) for t in rows.double().cpu().split(64, 1))
        want, _ = plain.decayed_attention(q, k, v, torch.tensor([0.0, 1.0]).double())
        close(out.view(n, 2, 32)[:, 0], want[:, 0], dtype)
        close(out.view(n, 2, 32)[:, 1], want[:, 1], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [64, 30, 2048])
def test_norm_before_the_gate(dtype, width):
    g = torch.Generator().manual_seed(8)
    y, z = ((4 * torch.randn(5, width + 8, generator=g)).to(dtype) for _ in range(2))
    weight = torch.randn(width, generator=g)
    out = torch.full((5, width + 8), 9.0, dtype=dtype, device="cuda")
    rlt.gated_norm(y.cuda()[:, :width], z.cuda()[:, :width], weight.cuda(), out[:, :width], 1, 1e-5, gate_behind=True)
    close(out[:, :width], plain.gated_output(y[:, :width].double(), z[:, :width].double(), weight.double(), 1e-5), dtype)
    assert bool((out[:, width:] == 9.0).all())


# ---- feed-forwards -------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["silu", "squared_relu"])
def test_further_activations(dtype, kind):
    x = torch.cat([torch.linspace(-90, 90, 4001), torch.linspace(-1e-3, 1e-3, 95)]).to(dtype).view(8, 512)
    out = torch.empty(8, 512, dtype=dtype, device="cuda")
    rlt.block_epilogue(x.cuda(), None, act=(0, 512, kind, out, 0))
    want = plain.silu(x.double()) if kind == "silu" else torch.relu(x.double()) ** 2
    assert bool(((out.double().cpu() - want).abs() <= {torch.bfloat16: 2.0 ** -8, torch.float32: 4e-6}[dtype] * want.abs() + 1e-6).all())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cols,up_col,limit", [(40, 40, 1.5), (33, 40, 0.7), (2048, 2048, 7.0)])
def test_clamped_unit(dtype, cols, up_col, limit):
    x = (4 * torch.randn(6, up_col + cols, generator=torch.Generator().manual_seed(2))).to(dtype)
    got = rlt.clamped_glu(x.cuda(), up_col, cols, limit, 1.702)
    close(got, plain.clamped_unit(x[:, :cols].double(), x[:, up_col:].double(), limit), dtype)


@pytest.mark.parametrize("rows,experts,top", [(1, 3, 3), (7, 9, 3), (200, 64, 8), (33, 40, 1), (5, 300, 6), (64, 1000, 32)])
def test_routing_chooses_by_corrected_and_weighs_by_plain_scores(rows, experts, top):
    g = torch.Generator().manual_seed(experts)
    logits, correction = 2 * torch.randn(rows, experts, generator=g), 0.05 * torch.randn(experts, generator=g)
    routing = rlt.expert_route(logits.cuda(), correction.cuda(), top)
    chosen, weights = plain.route(logits.double(), correction.double(), top)
    assert torch.equal(routing.chosen.cpu().long(), chosen)
    close(routing.weights, weights, torch.float32)
    assert torch.equal(routing.counts.cpu().long(), torch.bincount(chosen.flatten(), minlength=experts))
    ranks = {e: sorted(routing.rank.cpu()[chosen == e].tolist()) for e in range(experts)}
    assert all(r == list(range(len(r))) for r in ranks.values())
    uncorrected = rlt.expert_route(logits.cuda(), None, top)
    assert torch.equal(uncorrected.chosen.cpu().long(), plain.route(logits.double(), torch.zeros(experts).double(), top)[0])
    if rows == 200:
        assert not torch.equal(uncorrected.chosen, routing.chosen)


def test_equal_scores_take_the_lower_expert():
    routing = rlt.expert_route(torch.zeros(3, 70, device="cuda"), None, 4)
    assert routing.chosen.tolist() == [[0, 1, 2, 3]] * 3 and torch.allclose(routing.weights, torch.full((3, 4), 0.25, device="cuda"))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [96, 17])
def test_gathered_rows_are_sorted_by_expert(dtype, width):
    g = torch.Generator().manual_seed(1)
    x, logits = torch.randn(50, width, generator=g).to(dtype).cuda(), torch.randn(50, 7, generator=g).cuda()
    routing = rlt.expert_route(logits, None, 3)
    got = rlt.expert_gather(x, routing)
    places, chosen = routing.places.cpu(), routing.chosen.cpu()
    assert sorted(places.flatten().tolist()) == list(range(150))
    assert all(torch.equal(got[places[i, j]], x[i]) for i in range(50) for j in range(3))
    by_place = torch.empty(150, dtype=torch.int32)
    by_place[places.flatten().long()] = chosen.flatten()
    assert torch.equal(by_place, by_place.sort().values)


COUNTS = {"few": [3, 0, 1, 0, 0, 7, 2], "edges": [127, 128, 129, 0, 1, 256, 257], "one": [0, 0, 300, 0, 0, 0, 0], "tiny": [1] * 7, "many": [33] * 40 + [500]}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("act", [None, "squared_relu", "silu"])
@pytest.mark.parametrize("inner,outer", [(64, 128), (128, 72), (72, 136), (200, 264), (17, 9), (2048, 256), (8, 8)])
@pytest.mark.parametrize("counts", sorted(COUNTS))
def test_expert_products(dtype, act, inner, outer, counts):
    g = torch.Generator().manual_seed(inner)
    per = COUNTS[counts]
    x = torch.randn(sum(per), inner, generator=g).to(dtype).cuda()
    w = (torch.randn(len(per), outer, inner, generator=g) / inner ** 0.5).to(dtype).cuda()
    got = rlt.expert_gemm(x, w, torch.tensor(per, dtype=torch.int32, device="cuda"), act)
    want, at = [], 0
    for e, n in enumerate(per):
        want.append(x[at:at + n].double() @ w[e].double().T)
        at += n
    want = torch.cat(want)
    if act:
        want = plain.silu(want) if act == "silu" else torch.relu(want) ** 2
    close(got, want.cpu(), dtype, 2.0)


def test_the_mamba_scan_still_takes_its_own_decays():
    """Both forms of the recurrence share their kernels: driven by step sizes it is what it was."""
    g = torch.Generator().manual_seed(2)
    n, heads, groups, size, p = 150, 4, 2, 72, 40
    x, b, c, dt = (torch.randn(n, k, generator=g).bfloat16() for k in (heads * p, groups * size, groups * size, heads))
    bias, a_log, d = torch.randn(heads, generator=g), torch.linspace(-2, 1, heads), torch.randn(heads, generator=g)
    rows = torch.cat([x, b, c], 1).cuda()
    state, out = torch.zeros(1, heads, size, p, device="cuda"), torch.empty(n, heads * p, dtype=torch.bfloat16, device="cuda")
    at = heads * p, heads * p + groups * size
    rlt.ssd_scan(rows[:, :at[0]], rows[:, at[0]:at[1]], rows[:, at[1]:], dt.cuda(), bias.cuda(), a_log.cuda(), d.cuda(), state, out, group_of([n], [0], [0]))
    want, _ = plain_hybrid.recurrence(x.double().view(n, heads, p), b.double().view(n, groups, size), c.double().view(n, groups, size), dt.double(),
                                      bias.double(), a_log.double(), d.double())
    close(out.view(n, heads, p), want, torch.bfloat16)
