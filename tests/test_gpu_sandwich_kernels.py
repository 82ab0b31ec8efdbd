"""Each kernel of the decoder with norms on both sides of its sublayers alone against the plain float64 functions of plain_sandwich.py."""

from types import SimpleNamespace

import pytest
import torch

import plain_sandwich as plain
import vllm_rlt_b200 as rlt
from test_gpu_hybrid_kernels import BLOCK, DTYPES, close, paged_case, run_scored
from test_gpu_stream_kernels import latent_case, larger_pages, run_latent
from vllm_rlt_b200.engine import KeyRanges

pytestmark = pytest.mark.gpu


def generator(seed):
    return torch.Generator().manual_seed(seed)


# ---- the residual --------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,width", [(1, 33), (5, 52), (7, 96), (3, 1030), (4, 2048), (2, 4096), (3, 5001), (2, 12288)])
@pytest.mark.parametrize("centred", [True, False])
def test_residual_between_two_sublayers(dtype, rows, width, centred):
    g = generator(width)
    x, y = 2 + 3 * torch.randn(rows, width, generator=g), (1 + torch.randn(rows, width, generator=g)).to(dtype)
    before, behind = torch.randn(width, generator=g), torch.randn(width, generator=g)
    norm = plain.layer_norm if centred else plain.rms_norm
    want = x.double() + 0.7 * norm(y.double(), behind.double(), 1e-2)
    residual = x.cuda()
    h = rlt.residual_norm(residual, before.cuda(), 1e-2, dtype, delta=y.cuda(), behind=(behind.cuda(), 0.7), centred=centred)
    close(residual, want, torch.float32)
    close(h, norm(want, before.double(), 1e-2), dtype)
    index = torch.tensor([rows - 1, 0, rows - 1])
    residual = x.cuda()
    h = rlt.residual_norm(residual, before.cuda(), 1e-2, dtype, delta=y.cuda(), behind=(behind.cuda(), 0.7), centred=centred,
                          row_index=index.cuda(), store=False)
    assert torch.equal(residual.cpu(), x)
    close(h, norm(want[index], before.double(), 1e-2), dtype)
    h = rlt.residual_norm(residual, before.cuda(), 1e-2, dtype, delta=y.cuda(), centred=centred)         # no norm behind
    close(residual, x.double() + y.double(), torch.float32)
    close(h, norm(x.double() + y.double(), before.double(), 1e-2), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [33, 96])
def test_residual_starts_from_the_embedding(dtype, width):
    g = generator(1)
    embed, weight = torch.randn(13, width, generator=g).to(dtype), torch.randn(width, generator=g)
    tokens = torch.tensor([4, 0, 12, 4])
    residual = torch.full((4, width), float("nan"), device="cuda")
    h = rlt.residual_norm(residual, weight.cuda(), 1e-3, dtype, tokens=tokens.cuda(), embed=embed.cuda(), centred=True)
    assert torch.equal(residual.cpu(), embed[tokens].float())
    close(h, plain.layer_norm(embed[tokens].double(), weight.double(), 1e-3), dtype)


def test_a_layer_norm_far_from_zero_keeps_its_digits():
    """Mean 3000, deviation 1: sums of squares would lose what distinguishes the elements."""
    x = 3000 + torch.randn(3, 2048, generator=generator(2))
    h = rlt.residual_norm(x.cuda(), torch.ones(2048, device="cuda"), 1e-6, torch.float32, centred=True)
    error = (h.double().cpu() - plain.layer_norm(x.double(), 1.0, 1e-6)).abs().max()
    assert float(error) < 3e-4                              # the inputs' own spacing there is 2.4e-4


# ---- rotation ------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim,dims", [(16, 16), (64, 64), (24, 16), (10, 6), (11, 6), (2, 2), (40, 32)])
@pytest.mark.parametrize("scaling", [None, (8.0, 512, 16.0, 0.5)])
def test_halves_of_heads_turned_far_into_a_sequence(dtype, dim, dims, scaling):
    q = torch.randn(7, 3, 24 + dim, generator=generator(dim)).to(dtype)
    positions = torch.tensor([0, 1, 63, 1000, 65537, 1 << 20, 123456789], dtype=torch.int32)
    s = rlt.YarnScaling(*scaling) if scaling else None
    turns, amplitude = plain.frequencies(5e4, dims, dict(zip(("factor", "original", "fast", "slow"), scaling)) if scaling else None)
    frequencies, turn = rlt.rotation_frequencies(5e4, dims, "cuda", s), dict(halves=True, amplitude=s.amplitude if s else 1.0)
    want = q.double()
    want[:, :, 24:] = plain.rotate(want[:, :, 24:], positions, turns, amplitude)
    gpu, other = q.cuda(), torch.zeros(7, 3, dim, dtype=dtype, device="cuda")
    rlt.rotate_heads(gpu[:, :, 24:], other, frequencies, positions.cuda(), **turn)
    assert torch.equal(gpu.cpu(), q)
    rlt.rotate_heads(gpu[:, :, 24:], gpu[:, :, 24:], frequencies, positions.cuda(), **turn)
    close(gpu, want, dtype)
    assert torch.equal(other, gpu[:, :, 24:]) and torch.equal(other[:, :, dims:].cpu(), q[:, :, 24 + dims:])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("q_rank,kv_rank,rot_dim,dims", [(56, 48, 16, 16), (13, 11, 6, 6), (1536, 512, 64, 64), (8, 24, 12, 8), (24, 40, 5, 4),
                                                         (8, 16, 160, 144)])
def test_latent_rows_with_turned_halves(dtype, q_rank, kv_rank, rot_dim, dims):
    g = generator(3)
    rows, row = 5, kv_rank + rot_dim
    proj = (3 * torch.randn(rows, q_rank + 8 + row, generator=g)).to(dtype)
    wq, wk = torch.randn(q_rank, generator=g), torch.randn(kv_rank, generator=g)
    tables = torch.tensor([[4, 1], [0, 5]], dtype=torch.int32, device="cuda")
    positions = torch.tensor([15, 16, 0, 31, 3], dtype=torch.int32)
    batch = SimpleNamespace(tables=tables[None], row_seq=torch.tensor([0, 0, 1, 1, -1], dtype=torch.int32, device="cuda"), positions=positions.cuda())
    cache = torch.full((6, BLOCK, 1, row), 9.0, dtype=dtype, device="cuda")
    turns, _ = plain.frequencies(70.0, dims)
    rlt.latent_write(proj.cuda(), 0, q_rank + 8, wq.cuda(), wk.cuda(), 1e-3, rlt.rotation_frequencies(70.0, dims, "cuda"), cache, batch,
                     halves=True, amplitude=1.3)
    down = proj[:, q_rank + 8:].double()
    c, r = plain.rms_norm(down[:, :kv_rank], wk.double(), 1e-3), plain.rotate(down[:, kv_rank:], positions, turns, 1.3)
    for i, (page, slot) in enumerate([(4, 15), (1, 0), (0, 0), (5, 15)]):
        close(cache[page, slot, 0, :kv_rank], c[i], dtype)
        close(cache[page, slot, 0, kv_rank:], r[i], dtype)
        cache[page, slot] = 9.0
    assert bool((cache == 9.0).all())


# ---- convolution and unit norm in front of the scores --------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,taps", [(4, 2, 24, 40, 4), (3, 1, 10, 7, 1), (1, 1, 5, 3, 6), (8, 2, 128, 128, 3), (2, 2, 72, 136, 2),
                                                          (5, 5, 256, 64, 4), (2, 1, 16, 12, 33), (1, 1, 300, 20, 3), (6, 3, 128, 64, 4),
                                                          (2, 1, 32, 64, 1), (3, 3, 8, 8, 4)])
@pytest.mark.parametrize("unit_norm", [True, False])
def test_heads_behind_a_convolution(dtype, heads, kv_heads, dim, vdim, taps, unit_norm):
    """Two sequences in portions of unequal size, one of which starts late; pages, queries and the state that is carried on."""
    g = generator(taps + dim)
    widths = heads * dim, kv_heads * dim, kv_heads * vdim
    channels, columns = sum(widths), (8, 8 + widths[0] + (-widths[0]) % 8, 24 + widths[0] + (-widths[0]) % 8 + widths[1] + (-widths[1]) % 8)
    total = columns[2] + widths[2] + 5 + (-(columns[2] + widths[2] + 5)) % 8
    lengths = [75, 40]
    texts = [torch.randn(n, total, generator=g).to(dtype) for n in lengths]
    weight = torch.randn(channels, taps, generator=g)
    key = torch.full((8, BLOCK, kv_heads, dim), float("nan"), dtype=dtype, device="cuda")
    value = torch.full((8, BLOCK, kv_heads, vdim), float("nan"), dtype=dtype, device="cuda")
    tables = torch.tensor([[6, 2, 0, 7, 1], [3, 5, 4, -1, -1]], dtype=torch.int32)
    state = torch.full((4, taps - 1, channels), float("nan"), dtype=dtype, device="cuda")
    slots, at, got = [2, 0], [0, 0], [[], []]
    as_int = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    for portions in ([2, 0], [1, 1], [1, 3], [34, 33], [1, 1], [1, 1], [33, 1], [2, 0]):
        parts = [(s, n) for s, n in enumerate(portions) if n]
        rows = sum(n for _, n in parts)
        group = SimpleNamespace(sequences=len(parts), max_new=max(n for _, n in parts), cu=as_int([0, *torch.tensor([n for _, n in parts]).cumsum(0).tolist()]),
                                starts=as_int([at[s] for s, _ in parts]), lengths=as_int([at[s] + n for s, n in parts]), slots=as_int([slots[s] for s, _ in parts]),
                                tables=tables[[s for s, _ in parts]].contiguous().cuda())
        q = torch.empty(rows, heads, dim, dtype=dtype, device="cuda")
        rlt.conv_heads(torch.cat([texts[s][at[s]:at[s] + n] for s, n in parts]).cuda(), columns, weight.t().contiguous().cuda(), 1e-2, state, q, key, value, group, unit_norm=unit_norm)
        first = 0
        for s, n in parts:
            got[s].append(q[first:first + n])
            first, at[s] = first + n, at[s] + n
    assert at == lengths
    assert bool(state[1].isnan().all()) and bool(state[3].isnan().all())
    for s, n in enumerate(lengths):
        y = [plain.short_conv(texts[s][:, c:c + w].double(), part.double()) for c, w, part in zip(columns, widths, weight.split(widths))]
        wanted = [y[0].view(n, heads, dim), y[1].view(n, kv_heads, dim), y[2].view(n, kv_heads, vdim)]
        if unit_norm:
            wanted[:2] = [plain.rms_norm(x, 1.0, 1e-2) for x in wanted[:2]]
        paged = lambda cache: torch.stack([cache[tables[s, p // BLOCK], p % BLOCK] for p in range(n)])
        for have, want in zip((torch.cat(got[s]), paged(key), paged(value)), wanted):
            close(have, want, dtype)
        if taps > 1:
            last = torch.cat([texts[s][n - taps + 1:, c:c + w] for c, w in zip(columns, widths)], 1)
            assert torch.equal(state[slots[s]].cpu(), last)


@pytest.mark.parametrize("dtype", DTYPES)
def test_padding_rows_of_a_captured_step_write_no_page(dtype):
    key, value = (torch.full((3, BLOCK, 1, 16), 9.0, dtype=dtype, device="cuda") for _ in range(2))
    zero = torch.zeros(1, dtype=torch.int32, device="cuda")
    group = SimpleNamespace(sequences=1, max_new=1, cu=torch.tensor([0, 1], dtype=torch.int32, device="cuda"), starts=zero, lengths=zero,
                            slots=zero + 1, tables=torch.zeros(1, 2, dtype=torch.int32, device="cuda"))
    state = torch.full((2, 2, 48), 5.0, dtype=dtype, device="cuda")
    q = torch.empty(1, 1, 16, dtype=dtype, device="cuda")
    rlt.conv_heads(torch.ones(1, 48, dtype=dtype, device="cuda"), (0, 16, 32), torch.ones(3, 48, device="cuda"), 1e-5, state, q, key, value, group)
    assert bool((key == 9.0).all()) and bool((value == 9.0).all()) and bool((state[0] == 5.0).all()) and bool(torch.isfinite(q).all())


# ---- sinks ---------------------------------------------------------------------------------------
SINKS = torch.tensor([3.0, -60.0, 0.0, 80.0, 5.0, -2.0, 1.0])      # beside, far below and far above the scores


def sinks(heads):
    return SINKS.repeat(heads)[:heads].contiguous()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(4, 2, 24, 40), (8, 2, 128, 128), (7, 7, 64, 64), (3, 1, 9, 7)])
@pytest.mark.parametrize("window", [0, 40])
def test_scored_attention_with_sinks(dtype, heads, kv_heads, dim, vdim, window):
    terms = rlt.ScoreTerms(dim ** -0.5, window=window, sink=sinks(heads).cuda())
    for portions, contexts in (([1, 1, 3], [1, 130, 201]), ([1], [3000]), ([70, 150], [70, 230])):
        q, k, v, key, value, tables = paged_case(portions, contexts, heads, kv_heads, dim, vdim, dtype, 4)
        got = run_scored(q, key, value, tables, contexts, portions, terms, heads, dim, vdim)
        want = torch.cat([plain.attention(q[s].double(), k[s].double(), v[s].double(), dim ** -0.5, window, sinks(heads).double(),
                                          contexts[s] - portions[s]) for s in range(len(portions))])
        for h in range(heads):                   # a head whose sink takes nearly everything is compared with itself
            if SINKS[h % 7] < 50:
                close(got[:, h], want[:, h], dtype, 2.0)
            else:
                assert float(got[:, h].abs().max()) < 1e-20


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,rank,rot", [(6, 48, 16), (16, 512, 64), (5, 11, 6), (40, 128, 64)])
@pytest.mark.parametrize("window,page", [(0, 16), (0, 64), (70, 64)])
def test_attention_over_cache_rows_with_sinks(dtype, heads, rank, rot, window, page):
    row = rank + rot
    terms = rlt.ScoreTerms(0.7 * row ** -0.5, window=window, sink=sinks(heads).cuda())
    for portions, contexts in (([1, 1, 1], [1, 17, 530]), ([2, 16, 5], [2, 33, 300]), ([1], [64])):
        q, k, key, tables = latent_case(portions, contexts, heads, row, dtype, 7)
        if page > BLOCK:
            key, tables = larger_pages(key, tables, page)
        got = run_latent(q, key, tables, contexts, portions, rank, terms)
        want = torch.cat([plain.attention(q[s].double(), k[s].double()[:, None], k[s].double()[:, None, :rank], terms.scale, window,
                                          sinks(heads).double(), contexts[s] - portions[s]) for s in range(len(portions))])
        for h in range(heads):
            if SINKS[h % 7] < 50:
                close(got[:, h], want[:, h], dtype, 2.0)
            else:
                assert float(got[:, h].abs().max()) < 1e-20


def test_the_scale_leaves_a_sink_alone():
    """One key of score zero: the sink's share is exp(sink) / (1 + exp(sink)), whatever the scale."""
    for scale in (1e-3, 1.0, 30.0):
        for context in (1, 16):                  # equal keys: their weights add
            q, k = torch.zeros(1, 2, 16), torch.ones(context, 1, 16)
            key = k.view(1, -1, 1, 16) if context == 16 else torch.cat([k, torch.full((15, 1, 16), float("nan"))]).view(1, 16, 1, 16)
            terms = rlt.ScoreTerms(scale, sink=torch.tensor([0.0, 1.0], device="cuda"))
            got = run_scored([q], key, key, torch.zeros(1, 1, dtype=torch.int32), [context], [1], terms, 2, 16, 16)
            want = context / (context + torch.tensor([1.0, 2.718281828]))
            assert torch.allclose(got[0, :, 0].cpu(), want, rtol=1e-5)


def test_sinks_of_the_wrong_kind_are_refused():
    q, k, v, key, value, tables = paged_case([1], [5], 2, 1, 16, 16, torch.float32, 1)
    for sink in (torch.zeros(3, device="cuda"), torch.zeros(2, dtype=torch.bfloat16, device="cuda")):
        with pytest.raises(ValueError, match="sink"):
            run_scored(q, key, value, tables, [5], [1], rlt.ScoreTerms(1.0, sink=sink), 2, 16, 16)


# ---- prompts over packed keys and values ---------------------------------------------------------
PROMPTS = [([300], [300]), ([17, 64, 129], [17, 200, 129]), ([256, 257, 128], [300, 900, 128]), ([40, 600], [41, 600])]


def packed_case(portions, contexts, heads, kv_heads, dim, rot, vdim, window, seed, peak=None, sink=None, gate=None):
    """peak = distance: the last row of every portion finds the key that far back."""
    g = generator(seed)
    ranges = KeyRanges.of([(c - n, n) for c, n in zip(contexts, portions)], window, torch.device("cuda"))
    rand = lambda *shape: torch.randn(*shape, generator=g).bfloat16()
    q, k = [rand(n, heads, dim + rot) for n in portions], [rand(c, kv_heads, dim) for c in contexts]
    r, v = [rand(c, rot) for c in contexts], [rand(c, kv_heads, vdim) for c in contexts]
    if peak is not None:
        for s, c in enumerate(contexts):
            if c - 1 - peak >= 0:
                direction = torch.randn(dim, generator=g)
                direction /= direction.norm()
                q[s][-1, :, :dim] = (12 * direction).bfloat16()
                k[s][c - 1 - peak] = (12 * (dim + rot) ** 0.5 * direction).bfloat16()
    first, rows = ranges.first.tolist(), sum(portions)
    packed = lambda x: torch.cat([t[f:] for t, f in zip(x, first)]).cuda()
    out = torch.full((rows, heads, vdim), 7.0, dtype=torch.bfloat16, device="cuda")
    gates = None if gate is None else rand(rows, heads * (1 if gate == "head" else vdim) + 8)
    width = None if gate is None else gates.shape[1] - 8
    rlt.packed_attention(torch.cat(q).cuda(), packed(k), packed(v), out, ranges, (dim + rot) ** -0.5, window, shared_keys=packed(r) if rot else None,
                         sink=None if sink is None else sink.cuda(), gate=None if gate is None else gates.cuda()[:, :width])
    keys = [torch.cat([k[s], r[s][:, None].expand(-1, kv_heads, -1)], -1).double() for s in range(len(contexts))]
    want = torch.cat([plain.attention(q[s].double(), keys[s], v[s].double(), (dim + rot) ** -0.5, window, None if sink is None else sink.double(),
                                      contexts[s] - portions[s]) for s in range(len(contexts))]) if peak is None else v
    if gate is not None:
        want = want * plain.sigmoid(gates[:, :width].double()).view(rows, heads, -1)
    return out, want


@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(4, 2, 128, 128), (6, 2, 64, 80), (3, 1, 24, 40), (2, 2, 72, 24), (8, 1, 8, 128)])
@pytest.mark.parametrize("window", [1, 40, 64, 128, 129, 300, 0])
@pytest.mark.parametrize("portions,contexts", PROMPTS, ids=str)
def test_prompt_attention_of_grouped_heads(heads, kv_heads, dim, vdim, window, portions, contexts):
    got, want = packed_case(portions, contexts, heads, kv_heads, dim, 0, vdim, window, 3)
    close(got, want, torch.bfloat16, 2.0)


@pytest.mark.parametrize("heads,kv_heads,dim,rot,vdim", [(7, 7, 128, 64, 128), (4, 2, 64, 0, 80), (7, 1, 40, 8, 64)])
@pytest.mark.parametrize("gate", [None, "head", "element"])
@pytest.mark.parametrize("window", [0, 50])
def test_prompt_attention_with_sinks_and_gates(heads, kv_heads, dim, rot, vdim, gate, window):
    for portions, contexts in PROMPTS[1:3]:
        got, want = packed_case(portions, contexts, heads, kv_heads, dim, rot, vdim, window, 9, sink=sinks(heads), gate=gate)
        for h in range(heads):
            if SINKS[h % 7] < 50:
                close(got[:, h], want[:, h], torch.bfloat16, 2.0)
            else:
                assert float(got[:, h].abs().max()) < 1e-20


@pytest.mark.parametrize("window", [16, 64, 130, 200])
def test_grouped_prompt_rows_find_a_key_just_inside_the_window_and_none_outside(window):
    portions, contexts = [20, 150, 257, 129], [320, 333, 300, 400]
    for distance in (window - 1, window):
        got, v = packed_case(portions, contexts, 4, 2, 64, 0, 80, window, 5, peak=distance)
        at = 0
        for s, n in enumerate(portions):
            at += n
            value = v[s][contexts[s] - 1 - distance].double().repeat_interleave(2, 0)
            missed = float((got[at - 1].double().cpu() - value).norm() / value.norm())
            assert missed < 0.05 if distance < window else missed > 0.5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [16, 64, 130])
def test_decoded_rows_find_a_key_just_inside_the_window_and_none_outside(dtype, window):
    """Grouped heads over pages, one and several rows, at both sides of the window's edge and of pages."""
    for portions, contexts in (([1, 1, 1], [320, 257, 400]), ([2, 9, 16], [320, 333, 300])):
        for distance in (window - 1, window):
            peaks = [(s, n - 1, c - 1 - distance) for s, (n, c) in enumerate(zip(portions, contexts))]
            q, k, v, key, value, tables = paged_case(portions, contexts, 4, 2, 64, 80, dtype, 6, peaks=peaks)
            got = run_scored(q, key, value, tables, contexts, portions, rlt.ScoreTerms(64 ** -0.5, window=window), 4, 64, 80).double().cpu()
            at = 0
            for s, n in enumerate(portions):
                at += n
                wanted = v[s][contexts[s] - 1 - distance].double().repeat_interleave(2, 0)
                missed = float((got[at - 1] - wanted).norm() / wanted.norm())
                assert missed < 0.05 if distance < window else missed > 0.5


# ---- gates, units, caps --------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim", [(3, 40), (5, 7), (1, 1), (16, 128), (4, 1)])
@pytest.mark.parametrize("kind", ["head", "element"])
def test_gate_behind_the_heads(dtype, heads, dim, kind):
    g = generator(dim)
    y = torch.randn(6, heads, dim, generator=g).to(dtype)
    width = heads if kind == "head" else heads * dim
    gate = (4 * torch.randn(6, width + 16, generator=g)).to(dtype)
    want = y.double() * plain.sigmoid(gate[:, 8:8 + width].double()).view(6, heads, -1)
    gpu, view = y.cuda(), gate.cuda()[:, 8:8 + width]
    close(rlt.head_gate(gpu, view, torch.empty_like(gpu)), want, dtype)
    assert torch.equal(gpu.cpu(), y)
    rlt.head_gate(gpu, view)
    close(gpu, want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cols,up_col", [(40, 40), (33, 40), (2048, 2048)])
def test_gated_gelu_unit(dtype, cols, up_col):
    x = (2 * torch.randn(5, up_col + cols, generator=generator(cols))).to(dtype)
    x[0, :33] = torch.linspace(-30, 30, 33).to(dtype)
    got = rlt.gated_unit(x.cuda(), up_col, cols, "gelu_tanh")
    close(got, plain.gelu_tanh(x[:, :cols].double()) * x[:, up_col:up_col + cols].double(), dtype)


@pytest.mark.parametrize("shape", [(1, 1), (3, 131), (2, 2048)])
def test_soft_bound_on_logits(shape):
    x = 20 * torch.randn(shape, generator=generator(1))
    got = rlt.soft_cap(x.cuda(), 7.0)
    close(got, plain.soft_cap(x.double(), 7.0), torch.float32)
    assert float(got.abs().max()) <= 7.0
