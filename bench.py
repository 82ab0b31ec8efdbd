"""Benchmark of the self-speculative verify step on B200 (and its CPU baseline).

    python bench.py [--gpus N] [--steps K] [--warmup W] [--impl reference]

The contract line measures two things in one process per GPU.

1. Self-speculative decoding of an Ouro-1.4B-shaped model (24 layers, hidden 2048, 16 x 128 MHA,
   SwiGLU 5632, vocab 49152, 4 recurrent loops, random-init bf16): 128 concurrent requests with
   prompts of uniform-random tokens, lengths U[128, 1024], k = 4 drafts from loop depth 2 verified at
   depth 4, rejection sampling at temperature 0.8, through `SelfSpeculativeDecoder` /
   `B200SpeculativeRunner`.  A *step* is one speculative round of the whole batch (5 draft passes of
   128 rows through 2 loops, 2 verify passes of 640 rows, LM head, acceptance, rollback — one CUDA
   graph).  After the prompts are in the cache and the graph exists, W warm-up rounds run, then K
   rounds are timed with CUDA events (`value` = accepted tokens per second; committed tokens per
   second and the acceptance rate beside it), then K more rounds are timed on the host clock from
   `runner.submit(batch)` (Python request objects in) to `ticket.collect()` (Python token lists out):
   `e2e`.  The GEMMs of the model are cuBLAS call sites; every other kernel is this library's.
2. The verify attention alone at the kernel-microbench shape (64 requests, contexts U[512, 4096],
   16 rows per request = 4 tokens x 4 loop depths on a shared plane, 24-layer pool): its CUDA-event
   time per layer call against its algorithmic bytes is the `roofline` block, and its output for a
   few requests is compared with the CPU oracle (`parity`).

With N GPUs every rank is an independent engine replica that decodes the same 128 seeded requests
(no collective on the path); the timed regions are bracketed by a barrier, the step time is the
maximum over ranks and the tokens are summed, so the aggregate depends on step times only.

Other entry points (each prints its own JSON line; none is the contract line above):
    --workload decode [--requests R --output-tokens T --temperature X --k K --eager --prompt-min A --prompt-max B
                       --shared-prefix P --prefix-caching --in-flight F]
                      one complete generation (prompt pass included in `total_seconds`)
    --workload decode --engine reference [--sync]
                      the same requests, weights and output budget through the UNMODIFIED reference engine on the
                      GPU, when a copy of it is importable from baseline/_ref: its own scheduler, runner, Triton
                      attention and CUDA graphs (`ExecutionConfig(async_scheduling=True, cuda_graphs=True)`; greedy
                      only — `--sync` selects its synchronous runner, which also samples) — the same-box comparison;
                      `--adopt attention|runner` plugs this library's attention backend (and speculative runner) into
                      that engine (a backend name and a runner assignment on the reference's side)
    --workload sharded [--total-requests R ...]
                      R requests in total (default 1024, prompts U[256, 2048], 512 output tokens, k = 6, T = 0.8),
                      length-balanced over the ranks and decoded to completion in waves that fit the KV
                      pool: whole-job strong scaling
    --workload hybrid [--steps K --warmup W]
                      prefill and decode of Sobipel-shaped models (parallel attention / Mamba-2 blocks, random weights)
                      beside the looped model at equal size with one loop, through the same engine, and every kernel
                      of a layer against its roofline beside the like kernel of the looped model
    --workload stream [--steps K --warmup W]
                      the same for Sugosun-shaped models (hyper-connected streams, latent / lightning attention, dense and
                      mixture-of-experts feed-forwards)
    --workload sandwich [--steps K --warmup W]
                      the same for Kezuvik-shaped models (norms on both sides of a sublayer, latent attention with sinks and gates,
                      windowed attention behind a convolution), beside Sugosun and the looped model
    --only attention  [--requests --layers --tokens --depths --kv-heads --context-min --context-max --shared-plan]
    --only prefill    [--requests --tokens --kv-heads --eager]   packed causal prefill, TFLOP/s
    --only accept | --only silu                                  the small kernels at the step's shapes
"""

from __future__ import annotations

import argparse
import gc
import json
import os
import statistics
import subprocess
import sys
import time
from pathlib import Path

import torch

ROOT = Path(__file__).resolve().parent
if str(ROOT) not in sys.path:
    sys.path.insert(0, str(ROOT))

LAYERS, HEADS, HEAD_DIM, BLOCK, FFN, VOCAB = 24, 16, 128, 16, 5632, 49152
REQUESTS, TOKENS, DEPTHS = 64, 4, 4
TEMPERATURE = 0.8
DECODE_REQUESTS, DECODE_PROMPTS, DECODE_K, DECODE_OUTPUT = 128, (128, 1024), 4, 256
DRAFT_LOOPS, TARGET_LOOPS = 2, 4
METRIC = "accepted tokens/s/GPU, Ouro-1.4B self-spec decode; verify-attn % HBM peak"
# DRAM bytes (read + write) per algorithmic byte of verify_attention_kernel, from an ncu capture of a
# 32-request launch of the same kernel (654.4 + 7.9 MB moved for 653.9 MB algorithmic); traffic grows
# in proportion to the K/V read, so the ratio carries over to a full launch.
ATTENTION_TRAFFIC_RATIO = 1.0128


def measured_peaks():
    path = ROOT / "MEASURED_PEAKS.json"
    if path.exists():
        return float(json.loads(path.read_text())["hbm_gbs"]), "measured"
    return 6650.0, "fallback"


class Workload:
    """Seeded synthetic inputs of one replica (one GPU or the CPU sample)."""

    def __init__(self, seed: int, requests: int = REQUESTS, layers: int = LAYERS, device="cpu",
                 tokens: int = TOKENS, depths: int = DEPTHS, kv_heads: int = HEADS, context_range=(512, 4096)):
        g = torch.Generator().manual_seed(seed)
        self.requests, self.layers = requests, layers
        TOKENS, DEPTHS = tokens, depths
        self.kv_heads = kv_heads
        self.contexts = torch.randint(context_range[0], context_range[1] + 1, (requests,), generator=g)
        pages = (self.contexts + BLOCK - 1) // BLOCK
        self.total_pages = int(pages.sum())
        order = torch.randperm(self.total_pages, generator=g).int()
        width = int(pages.max())
        tables = torch.zeros(requests, width, dtype=torch.int32)
        offset = 0
        for i, n in enumerate(pages.tolist()):
            tables[i, :n] = order[offset:offset + n]
            offset += n
        self.request_tables = tables
        rows_per_request = TOKENS * DEPTHS
        # row (depth, t) of a request sees ctx - 3 + t keys; all 16 rows share one table row
        visible = torch.stack([self.contexts - (TOKENS - 1) + t for t in range(TOKENS)], 1)  # [req, tok]
        self.lengths = visible.repeat(1, DEPTHS).reshape(-1).int()
        self.tables = tables.repeat_interleave(rows_per_request, 0).contiguous()
        self.rows = requests * rows_per_request
        positions = (visible - 1).reshape(-1)  # new tokens: one K/V row per (request, token)
        req_of = torch.arange(requests).repeat_interleave(TOKENS)
        self.write_blocks = tables[req_of, (positions // BLOCK)].long()
        self.write_offsets = (positions % BLOCK).long()
        self.kv_rows = requests * TOKENS
        self.seed = seed
        self.device = torch.device(device)
        self.generator = g
        # acceptance inputs: 4 rows per request (3 drafts + bonus row)
        self.accept_rows = requests * TOKENS
        self.cu_rows = (torch.arange(requests + 1) * TOKENS).int()
        self.starts = (self.contexts - TOKENS).long()
        self.slots = torch.randperm(2 * requests, generator=g)[:requests]
        self.temperature = torch.full((requests,), TEMPERATURE)

    def algorithmic_attention_bytes(self) -> int:
        """Each group's K/V once + Q + O + block tables, per layer call."""
        kv = int(self.contexts.sum()) * self.kv_heads * HEAD_DIM * 2 * 2
        qo = self.rows * HEADS * HEAD_DIM * 2 * 2
        tables = int(((self.contexts + BLOCK - 1) // BLOCK).sum()) * 4
        return kv + qo + tables

    def host_inputs(self, pin: bool):
        """Per-step inputs as host tensors (bf16 activations, fp32 logits)."""
        g = self.generator
        def mk(*shape, scale=1.0, dtype=torch.bfloat16):
            t = (torch.randn(*shape, generator=g) * scale).to(dtype)
            return t.pin_memory() if pin else t
        inputs = dict(
            q=mk(self.layers, self.rows, HEADS, HEAD_DIM, scale=0.5),
            k=mk(self.layers, self.kv_rows, HEADS, HEAD_DIM, scale=0.5),
            v=mk(self.layers, self.kv_rows, HEADS, HEAD_DIM, scale=0.5),
            gate=mk(self.layers, self.rows, FFN, scale=3.0),
            up=mk(self.layers, self.rows, FFN),
            target=mk(self.accept_rows, VOCAB, scale=3.0, dtype=torch.float32),
        )
        noise = mk(self.accept_rows, VOCAB, scale=0.5, dtype=torch.float32)
        draft = inputs["target"] + noise
        inputs["draft"] = draft.pin_memory() if pin else draft
        small = dict(tables=self.tables, lengths=self.lengths, write_blocks=self.write_blocks,
                     write_offsets=self.write_offsets, cu_rows=self.cu_rows, starts=self.starts,
                     slots=self.slots, temperature=self.temperature,
                     u_draft=torch.rand(self.accept_rows, generator=g),
                     u_accept=torch.rand(self.accept_rows, generator=g),
                     u_final=torch.rand(self.requests, generator=g),
                     request_tables=self.request_tables[:, None, :].repeat(1, DEPTHS, 1).contiguous())
        for name, t in small.items():
            inputs[name] = t.pin_memory() if pin else t
        return inputs


def combine_ranks(stats, world: int, steps: int, gather=None):
    """Whole-job numbers from per-rank [timed ms, e2e ms, accepted/step, committed/step].

    Replicas are independent, so the job's step time is the slowest rank's (max over ranks) and its
    tokens are the sum over ranks.  `gather(tensor) -> [world, 4]` collects the rows
    (torch.distributed all_gather in a multi-rank run)."""
    if stats.dim() == 2:
        table = stats                                      # already one row per rank
    else:
        table = stats[None] if gather is None or world == 1 else gather(stats)
    max_ms, max_e2e_ms = float(table[:, 0].max()), float(table[:, 1].max())
    accepted, committed = float(table[:, 2].sum()), float(table[:, 3].sum())
    ms_per_step = max_ms / steps
    return {
        "ms_per_step": ms_per_step,
        "e2e_ms_per_step": max_e2e_ms / steps,
        "accepted_per_step": accepted,
        "committed_per_step": committed,
        "accepted_tokens_per_s": accepted / (ms_per_step / 1e3),
        "committed_tokens_per_s": committed / (ms_per_step / 1e3),
        "e2e_accepted_tokens_per_s": accepted / (max_e2e_ms / steps / 1e3),
    }


def all_gather_rows(stats):
    """[4] per rank -> [world, 4] on every rank (any torch.distributed backend)."""
    import torch.distributed as dist

    rows = [torch.zeros_like(stats) for _ in range(dist.get_world_size())]
    dist.all_gather(rows, stats)
    return torch.stack(rows).cpu()


def replica_seed(rank: int) -> int:
    """Every replica draws its own requests: same distribution, different seed."""
    return 1234 + rank


class ClockSampler:
    """Samples nvidia-smi clocks and throttle reasons while the timed region runs."""

    QUERY = ("index,clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.active,"
             "clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
             "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self, index: int):
        try:  # address the GPU by UUID: nvidia-smi indices ignore CUDA_VISIBLE_DEVICES
            index = "GPU-" + str(torch.cuda.get_device_properties(index).uuid)
        except Exception:
            pass
        self.index, self.samples, self.process = index, [], None

    def __enter__(self):
        try:
            self.process = subprocess.Popen(
                ["nvidia-smi", f"--id={self.index}", f"--query-gpu={self.QUERY}", "--format=csv,noheader,nounits",
                 "-lms", "50"], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
        except Exception:
            self.process = None
        return self

    def __exit__(self, *exc):
        if self.process is None:
            return
        self.process.terminate()
        try:
            out, _ = self.process.communicate(timeout=5)
        except Exception:
            self.process.kill()
            out = ""
        for line in out.splitlines():
            fields = [x.strip() for x in line.split(",")]
            if len(fields) >= 9:
                self.samples.append(fields)

    def summary(self):
        sm = [float(s[1]) for s in self.samples if len(s) > 2 and s[1].replace(".", "").isdigit()]
        mx = [float(s[2]) for s in self.samples if len(s) > 2 and s[2].replace(".", "").isdigit()]
        reasons = set()
        names = ("hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap")
        for s in self.samples:
            for name, flag in zip(names, s[5:9]):
                if flag.lower().startswith("active"):
                    reasons.add(name)
        return {"sm_mhz": statistics.median(sm) if sm else None, "sm_max_mhz": max(mx) if mx else None,
                "reasons": sorted(reasons), "samples": len(self.samples)}


def decode_prompts(requests: int, prompt_range, vocab: int, seed: int = 11):
    """Uniform-random token prompts with lengths U[prompt_range] (the same list for a given seed)."""
    g = torch.Generator().manual_seed(seed)
    lengths = torch.randint(prompt_range[0], prompt_range[1] + 1, (requests,), generator=g).tolist()
    return [torch.randint(1, vocab, (n,), generator=g).tolist() for n in lengths]


def decode_round_bytes(config, stats_before, stats_after, rounds: int, k: int):
    """Algorithmic HBM bytes of `rounds` speculative rounds: every recurrent pass streams the layer
    weights once and, per layer, the K/V of every context it attends to once per request; every LM-head
    call streams lm_head once (k draft calls and one verify call per round).  Activations and logits are
    left out (a few percent)."""
    c = config
    layer_params = (c.hidden_size * (c.num_attention_heads + 2 * c.num_key_value_heads) * c.head_dim
                    + c.num_attention_heads * c.head_dim * c.hidden_size + 3 * c.hidden_size * c.intermediate_size)
    passes = stats_after.loop_passes - stats_before.loop_passes
    context_tokens = stats_after.context_tokens_read - stats_before.context_tokens_read
    weight_bytes = 2.0 * c.num_hidden_layers * layer_params * passes
    kv_bytes = 2.0 * 2 * c.num_key_value_heads * c.head_dim * c.num_hidden_layers * context_tokens
    head_bytes = 2.0 * c.vocab_size * c.hidden_size * (k + 1) * rounds
    return {"weight_bytes": weight_bytes, "kv_bytes": kv_bytes, "lm_head_bytes": head_bytes,
            "total": weight_bytes + kv_bytes + head_bytes}


def launches_per_round(config, k: int, draft_loops: int, target_loops: int, sampled: bool) -> int:
    """Kernels of this library in one round's graph (the cuBLAS GEMMs and the small index kernels of
    the host layer are not counted): per recurrent pass one attention plan, one opening norm and per
    layer rope_kv_write, attention + merge, SiLU-and-Mul and two sandwich norms; per draft offset one
    proposal kernel; acceptance (two launches), the round's uniforms when sampling, rollback."""
    passes = draft_loops * (k + 1) + target_loops - draft_loops
    per_pass = 2 + 6 * config.num_hidden_layers
    return passes * per_pass + k + 2 + (1 if sampled else 0) + 1


def copy_stats(stats):
    import copy

    return copy.copy(stats)


def attention_roofline(device, steps: int, warmup: int, parity_requests: int):
    """The verify attention at the kernel-microbench shape inside a 24-layer pass (KV write ->
    attention -> SiLU-and-Mul per layer, one plan per pass): CUDA-event time per attention call, its
    algorithmic bytes, and a comparison of layer 0's output for `parity_requests` requests with the
    CPU oracle.  Returns (roofline dict, parity dict, launches)."""
    import vllm_rlt_b200 as rlt

    work = Workload(seed=1234)
    g = torch.Generator(device=device).manual_seed(99)
    pool_shape = (work.total_pages, LAYERS, BLOCK, HEADS, HEAD_DIM)
    key_pool = torch.empty(pool_shape, dtype=torch.bfloat16, device=device)
    value_pool = torch.empty(pool_shape, dtype=torch.bfloat16, device=device)
    for pool in (key_pool, value_pool):  # N(0,1) * 0.5, generated in slabs to bound temporaries
        flat = pool.view(-1)
        slab = 1 << 28
        for start in range(0, flat.numel(), slab):
            n = min(slab, flat.numel() - start)
            flat[start:start + n] = (torch.randn(n, device=device, generator=g) * 0.5).to(torch.bfloat16)

    def mk(*shape, scale=1.0):
        return (torch.randn(*shape, device=device, generator=g) * scale).to(torch.bfloat16)

    q = mk(LAYERS, work.rows, HEADS, HEAD_DIM, scale=0.5)
    k_new = mk(LAYERS, work.kv_rows, HEADS, HEAD_DIM, scale=0.5)
    v_new = mk(LAYERS, work.kv_rows, HEADS, HEAD_DIM, scale=0.5)
    gate, up = mk(work.rows, FFN, scale=3.0), mk(work.rows, FFN)
    tables, lengths = work.tables.to(device), work.lengths.to(device)
    write_blocks, write_offsets = work.write_blocks.to(device), work.write_offsets.to(device)
    backend = rlt.create_backend(device, torch.bfloat16, HEAD_DIM, BLOCK)
    events, launches, first_out = [], 0, None
    for step in range(warmup + steps):
        with backend.kernel.shared_plan():
            for layer in range(LAYERS):
                kc, vc = key_pool[:, layer], value_pool[:, layer]
                rlt.kv_write(kc, vc, k_new[layer], v_new[layer], write_blocks, write_offsets)
                a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                a.record()
                out = backend(q[layer], kc, vc, tables, lengths)
                b.record()
                rlt.silu_and_mul(gate, up)
                if step >= warmup:
                    events.append((a, b))
                    launches += 4
                if step == 0 and layer == 0:
                    first_out = out
        launches += 1 if step >= warmup else 0
    torch.cuda.synchronize()
    attention_ms = statistics.mean(a.elapsed_time(b) for a, b in events)
    status = backend.kernel.last_status(device)
    peak, peak_kind = measured_peaks()
    algorithmic = work.algorithmic_attention_bytes()
    achieved = algorithmic / (attention_ms * 1e-3) / 1e9
    roofline = {"bound": "hbm", "kernel": "verify_attention_kernel + merge_kernel, per layer call of a 24-layer pass "
                                          "(64 requests, ctx U[512,4096], 16 rows per request on a shared plane; "
                                          "inputs larger than L2: 34 GB pool streamed once per pass)",
                "achieved": achieved, "peak": peak, "peak_kind": peak_kind, "unit": "GB/s", "frac": achieved / peak,
                "traffic": ATTENTION_TRAFFIC_RATIO * algorithmic,
                "traffic_source": "ncu dram bytes of a 32-request launch scaled by algorithmic bytes",
                "algorithmic_bytes": algorithmic, "avg_launch_ms": attention_ms, "timed_calls": len(events),
                "attention_status": status}
    parity = attention_parity(work, first_out, q[0], key_pool, value_pool, parity_requests)
    return roofline, parity, launches


def attention_parity(work, gpu_out, q0, key_pool, value_pool, requests: int):
    """Layer 0 of the full-size microbench against the CPU oracle for the first `requests` requests:
    their pages are copied to the host (with the new tokens' K/V already written), renumbered, and the
    oracle scores the same 16 rows per request.  Tolerance: 2e-2 absolute + 2e-2 relative (bf16)."""
    from oracle import oracle

    rows_per_request = TOKENS * DEPTHS
    pages = ((work.contexts + BLOCK - 1) // BLOCK)[:requests]
    ids = torch.cat([work.request_tables[i, : int(n)] for i, n in enumerate(pages.tolist())]).long()
    kc = key_pool[ids.to(key_pool.device), 0].cpu()
    vc = value_pool[ids.to(key_pool.device), 0].cpu()
    tables = torch.zeros(requests * rows_per_request, int(pages.max()), dtype=torch.int32)
    offset = 0
    for i, n in enumerate(pages.tolist()):
        tables[i * rows_per_request:(i + 1) * rows_per_request, :n] = torch.arange(offset, offset + n, dtype=torch.int32)
        offset += n
    rows = requests * rows_per_request
    want = oracle.paged_attention(q0[:rows].cpu(), kc, vc, tables, work.lengths[:rows]).float()
    got = gpu_out[:rows].float().cpu()
    diff = (got - want).abs()
    bound = 2e-2 + 2e-2 * want.abs()
    return {"against": "CPU oracle", "requests": requests, "rows": rows, "max_abs": float(diff.max()),
            "max_rel_of_bound": float((diff / bound).max()), "tolerance": "2e-2 abs + 2e-2 rel (bf16)",
            "ok": bool((diff <= bound).all())}


def run_gpu(args):
    import torch.distributed as dist

    import vllm_rlt_b200 as rlt

    rank = int(os.environ.get("RANK", "0"))
    world = int(os.environ.get("WORLD_SIZE", "1"))
    local = int(os.environ.get("LOCAL_RANK", "0"))
    torch.cuda.set_device(local)
    device = torch.device("cuda", local)
    if world > 1:
        dist.init_process_group("nccl", device_id=device)

    def barrier():
        if world > 1:
            dist.barrier()
        torch.cuda.synchronize()

    # ---- 1. the verify attention alone (roofline + parity), rank 0 ---------------------------
    roofline = parity = None
    attention_launches = 0
    if rank == 0:
        roofline, parity, attention_launches = attention_roofline(device, steps=min(args.steps, 10), warmup=2,
                                                                  parity_requests=4)
        gc.collect()
        torch.cuda.empty_cache()

    # ---- 2. self-speculative decoding: K rounds on the device clock, K on the host clock ------
    steps, warmup = args.steps, args.warmup
    k = DECODE_K
    e2e_warmup = min(warmup, 3)
    rounds_needed = warmup + steps + e2e_warmup + steps + 2
    max_tokens = max(DECODE_OUTPUT, rounds_needed * (k + 1))
    config = rlt.LoopedLMConfig()
    model = rlt.LoopedLM(config, rlt.seeded_state_dict(config, 3, device=device), device, torch.bfloat16)
    prompts = decode_prompts(DECODE_REQUESTS, DECODE_PROMPTS, config.vocab_size)
    decoder = rlt.SelfSpeculativeDecoder(model, cuda_graphs=True, capture_sizes=[DECODE_REQUESTS])
    torch.cuda.synchronize()
    t_open = time.perf_counter()
    session = decoder.open(prompts, max_tokens, num_speculative_tokens=k, draft_loops=DRAFT_LOOPS,
                           target_loops=TARGET_LOOPS, temperature=TEMPERATURE, seed=1, in_flight=2)
    torch.cuda.synchronize()
    open_seconds = time.perf_counter() - t_open
    stats = decoder.stats

    def run_rounds(count):
        """`count` rounds, two in flight, every one collected before this returns."""
        submitted = collected = 0
        while collected < count:
            while submitted < count and session.submit_round():
                submitted += 1
            if not session.collect_round():
                raise RuntimeError("the requests ran out of output budget inside the timed region")
            collected += 1

    run_rounds(warmup)
    barrier()
    clocks = ClockSampler(local)
    clocks.__enter__()
    before = copy_stats(stats)
    start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    start.record()
    run_rounds(steps)
    stop.record()
    barrier()
    device_ms = start.elapsed_time(stop)
    after = copy_stats(stats)
    accepted = after.accepted_tokens - before.accepted_tokens
    committed = after.committed_tokens - before.committed_tokens
    drafted = after.drafted_tokens - before.drafted_tokens
    round_bytes = decode_round_bytes(config, before, after, steps, k)

    run_rounds(e2e_warmup)
    barrier()
    before_e2e = copy_stats(stats)
    t0 = time.perf_counter()
    run_rounds(steps)
    torch.cuda.synchronize()
    e2e_ms = (time.perf_counter() - t0) * 1e3
    barrier()
    clocks.__exit__(None, None, None)
    after_e2e = copy_stats(stats)
    e2e_accepted = after_e2e.accepted_tokens - before_e2e.accepted_tokens
    runner = decoder.runner
    nb, w = runner.bucket_of(DECODE_REQUESTS), runner.width
    h2d, d2h = 3 * nb * 8, (nb * w + 4 * nb) * 8
    decode_status = model.attention.last_status(device)
    tokens_host = sum(len(r.generated_token_ids) for r in session.requests)

    times = torch.tensor([device_ms, e2e_ms, float(accepted), float(committed), float(e2e_accepted), float(drafted)],
                         dtype=torch.float64, device=device)
    table = times[None].cpu() if world == 1 else all_gather_rows(times)
    if rank == 0:
        per_step = table[:, :4].clone()
        per_step[:, 2:] /= steps                         # tokens of the timed window -> per step
        job = combine_ranks(per_step, world, steps)
        max_ms, mean_ms = float(table[:, 0].max()), float(table[:, 0].mean())
        e2e_value = float(table[:, 4].sum()) / (float(table[:, 1].max()) / 1e3)
        peak, peak_kind = measured_peaks()
        seconds = device_ms / 1e3
        per_round = launches_per_round(config, k, DRAFT_LOOPS, TARGET_LOOPS, True)
        line = {
            "metric": METRIC, "value": job["accepted_tokens_per_s"], "unit": "accepted tokens/s", "n_gpus": world,
            "steps": steps, "warmup": warmup, "ms_per_step": job["ms_per_step"],
            "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16",
            "data": "synthetic",
            "config": {
                "workload": "configs[2]: Ouro-1.4B-shaped random-init bf16 model (24 layers, hidden 2048, 16x128 MHA, "
                            "FFN 5632, vocab 49152, 4 loops), 128 concurrent requests per GPU, prompts U[128,1024] of "
                            "uniform-random tokens, self-speculation k=4 from depth 2 verified at depth 4, rejection "
                            "sampling T=0.8; step = one speculative round of the whole batch (one CUDA graph), timed "
                            "in steady state after the prompt pass; roofline block: configs[1] verify attention",
                "requests_per_gpu": DECODE_REQUESTS, "k": k, "draft_loops": DRAFT_LOOPS, "target_loops": TARGET_LOOPS,
                "temperature": TEMPERATURE, "output_budget_tokens": max_tokens, "rounds_in_flight": 2,
                "kv_pool_gb": round(2 * session.runner.cache.key.numel() * 2 / 1e9, 2),
                "l2_policy": "inputs larger than L2 (every pass streams the active contexts' K/V and the layer weights)",
                "parallelism": f"{world} independent replicas decoding the same seeded requests, no collective",
                "prompt_pass_and_graph_capture_seconds": open_seconds,
            },
            "committed_tokens_per_s": job["committed_tokens_per_s"],
            "acceptance_rate": float(table[:, 2].sum()) / max(float(table[:, 5].sum()), 1.0),
            "accepted_per_step": job["accepted_per_step"], "committed_per_step": job["committed_per_step"],
            "rank_time_imbalance_max_over_mean": max_ms / mean_ms,
            "e2e": {"value": e2e_value, "unit": "accepted tokens/s", "h2d_bytes_per_step": h2d,
                    "d2h_bytes_per_step": d2h, "ms_per_step": float(table[:, 1].max()) / steps,
                    "path": "runner.submit(Python requests) -> graph replay -> ticket.collect() -> Python token lists, "
                            "host clock", "tokens_on_host": tokens_host},
            "gpu_launches": per_round * steps,
            "hbm_roofline_decode": {**round_bytes, "peak_gbs": peak, "peak_kind": peak_kind,
                                    "seconds_at_peak": round_bytes["total"] / (peak * 1e9),
                                    "frac": round_bytes["total"] / (peak * 1e9) / seconds},
            "roofline": roofline, "parity": parity,
            "clocks": clocks.summary(),
            "attention_status": decode_status,
        }
        if not args.no_cpu_baseline and world == 1:
            del session, decoder, model, runner
            gc.collect()
            torch.cuda.empty_cache()
            line["cpu_baseline"] = cpu_baseline(threads=os.cpu_count() or 1, rounds=2)
        print(json.dumps(line))
    if world > 1:
        dist.destroy_process_group()


def run_attention_only(args):
    """Profiling aid: only the verify-attention calls of `--layers` layers for `--requests` requests
    (same shapes and seeds as the full step), timed per call with CUDA events.  Prints one JSON line."""
    import vllm_rlt_b200 as rlt

    torch.cuda.set_device(0)
    device = torch.device("cuda", 0)
    work = Workload(seed=1234, requests=args.requests, layers=args.layers, tokens=args.tokens, depths=args.depths,
                    context_range=(args.context_min, args.context_max),
                    kv_heads=args.kv_heads)
    g = torch.Generator(device=device).manual_seed(99)
    pool_shape = (work.total_pages, args.layers, BLOCK, args.kv_heads, HEAD_DIM)
    key_pool = (torch.randn(pool_shape, device=device, generator=g) * 0.5).to(torch.bfloat16)
    value_pool = (torch.randn(pool_shape, device=device, generator=g) * 0.5).to(torch.bfloat16)
    q = (torch.randn(args.layers, work.rows, HEADS, HEAD_DIM, device=device, generator=g) * 0.5).to(torch.bfloat16)
    tables, lengths = work.tables.to(device), work.lengths.to(device)
    backend = rlt.create_backend(device, torch.bfloat16, HEAD_DIM, BLOCK)
    events = []
    from contextlib import nullcontext
    for step in range(args.warmup + args.steps):
        with backend.kernel.shared_plan() if args.shared_plan else nullcontext():
            for layer in range(args.layers):
                a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                a.record()
                backend(q[layer], key_pool[:, layer], value_pool[:, layer], tables, lengths)
                b.record()
                if step >= args.warmup:
                    events.append((a, b))
    torch.cuda.synchronize()
    ms = statistics.mean(a.elapsed_time(b) for a, b in events)
    peak, kind = measured_peaks()
    algorithmic = work.algorithmic_attention_bytes()
    print(json.dumps({"only": "attention", "requests": args.requests, "layers": args.layers, "rows": work.rows,
                      "avg_call_ms": ms, "algorithmic_bytes": algorithmic,
                      "achieved_gbs": algorithmic / ms / 1e6, "frac": algorithmic / ms / 1e6 / peak,
                      "peak_kind": kind, "status": backend.kernel.last_status(device)}))


def run_prefill_only(args):
    """Profiling aid (`--only prefill`): packed causal prefill of `--requests` prompts of `--tokens`
    tokens each (16 x 128 MHA, bf16, 16-token pages, pages in random order) through
    `AttentionBackend.prefill`, timed per call with CUDA events.  Tensor-bound: reports TFLOP/s
    (4 * head_dim flops per visible (query, key) pair and head) against the measured bf16 peak."""
    import vllm_rlt_b200 as rlt

    torch.cuda.set_device(0)
    device = torch.device("cuda", 0)
    g = torch.Generator(device=device).manual_seed(17)
    n, seqs = args.tokens, args.requests
    pages = -(-n // BLOCK)
    total = pages * seqs
    shape = (total, 1, BLOCK, args.kv_heads, HEAD_DIM)
    both = (torch.randn((2,) + shape, device=device, generator=g) * 0.5).to(torch.bfloat16)
    key, value = both[0][:, 0], both[1][:, 0]
    tables = torch.randperm(total, device=device, generator=g).int().view(seqs, pages)
    lengths = torch.full((seqs,), n, dtype=torch.int32, device=device)
    cu = (torch.arange(seqs + 1, device=device) * n).int()
    q = (torch.randn(seqs * n, HEADS, HEAD_DIM, device=device, generator=g) * 0.5).to(torch.bfloat16)
    kernel = rlt.B200PagedAttention()
    max_new = n if not args.eager else 0          # --eager: the same rows through the grouped verify kernel
    for _ in range(args.warmup):
        kernel.prefill(q, key, value, tables, lengths, cu, max_new)
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(args.steps):
        kernel.prefill(q, key, value, tables, lengths, cu, max_new)
    b.record()
    torch.cuda.synchronize()
    ms = a.elapsed_time(b) / args.steps
    flops = 4.0 * HEAD_DIM * HEADS * seqs * (n * (n + 1) / 2)
    peaks = json.loads((ROOT / "MEASURED_PEAKS.json").read_text()) if (ROOT / "MEASURED_PEAKS.json").exists() else {}
    peak = float(peaks.get("bf16_tflops", 1590.0))
    print(json.dumps({"only": "prefill", "kernel": "grouped verify kernel" if args.eager else "prefill kernel",
                      "sequences": seqs, "tokens": n, "kv_heads": args.kv_heads, "ms_per_call": ms,
                      "algorithmic_flops": flops, "tflops": flops / ms / 1e9, "peak_tflops": peak,
                      "peak_kind": "measured" if peaks else "fallback", "frac": flops / ms / 1e9 / peak}))


def silu_comparison(device, steps: int, warmup: int):
    """SiLU-and-Mul at the path's shapes, this library's kernel beside the reference's own CUDA kernel when its
    extension (`vllm_rlt._C`, built from the reference's unmodified csrc for sm_100) is present under
    baseline/_ref: CUDA events, per call, L2-warm (the same tensors every call) and L2-cold (a ring of input
    sets larger than L2, so every call reads from HBM), plus one case where gate, up and out each start at a
    different 16-byte misalignment."""
    import glob

    import vllm_rlt_b200 as rlt

    kernels = {"b200": rlt.silu_and_mul}
    found = glob.glob(str(ROOT / "baseline" / "_ref" / "vllm_rlt" / "_C*.so"))
    note = None
    if found:
        try:
            torch.ops.load_library(found[0])
            kernels["reference"] = torch.ops.vllm_rlt.silu_and_mul
        except Exception as error:
            note = f"the reference extension did not load: {error}"
    else:
        note = "no reference extension under baseline/_ref"
    g = torch.Generator(device=device).manual_seed(3)
    peak, _ = measured_peaks()

    unroll = 32

    def timed(fn, sets):
        """Microseconds per call: a CUDA graph of `unroll` calls (as the reference's own benchmark of this
        kernel does, benchmarks/kernels/silu_and_mul.py there), replayed `steps` times, so that the host's
        per-call cost is not what is measured."""
        for i in range(max(warmup, 1)):
            fn(*sets[i % len(sets)])
        torch.cuda.synchronize()
        calls = max(unroll, len(sets))                 # every set of a cold ring is visited once per replay
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            kept = [fn(*sets[i % len(sets)]) for i in range(calls)]
        graph.replay()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        for _ in range(max(steps, 1)):
            graph.replay()
        b.record()
        torch.cuda.synchronize()
        del kept
        return a.elapsed_time(b) / (max(steps, 1) * calls) * 1e3

    table = []
    for rows in (128, 640, 768, 1024):
        nbytes = 3 * rows * FFN * 2
        ring = max(2, int(400e6 // (2 * rows * FFN * 2)) + 1)            # inputs of the ring: > 3 x L2
        sets = [((torch.randn(rows, FFN, device=device, generator=g) * 3).to(torch.bfloat16),
                 torch.randn(rows, FFN, device=device, generator=g).to(torch.bfloat16)) for _ in range(ring)]
        row = {"shape": [rows, FFN], "dtype": "bf16", "bytes": nbytes}
        for name, fn in kernels.items():
            warm, cold = timed(fn, sets[:1]), timed(fn, sets)
            row[name] = {"warm_us": warm, "cold_us": cold, "cold_gbs": nbytes / cold / 1e3, "cold_frac": nbytes / cold / 1e3 / peak}
        if "reference" in kernels:
            assert torch.equal(kernels["b200"](*sets[0]), kernels["reference"](*sets[0]))
        table.append(row)
        del sets
    # independent misalignments: gate +2, up +4, (out is allocated by the op) elements off a 16-byte boundary
    rows = 640
    base = [torch.randn(rows * FFN + 16, device=device, generator=g).to(torch.bfloat16) for _ in range(2)]
    gate, up = base[0][1:1 + rows * FFN].view(rows, FFN), base[1][2:2 + rows * FFN].view(rows, FFN)
    row = {"shape": [rows, FFN], "dtype": "bf16", "misaligned": "gate +2 bytes, up +4 bytes", "bytes": 3 * rows * FFN * 2}
    for name, fn in kernels.items():
        row[name] = {"warm_us": timed(fn, [(gate, up)])}
    table.append(row)
    return {"silu_and_mul": table, "reference_kernel": "vllm_rlt._C built from the reference's csrc for sm_100"
            if "reference" in kernels else None, "note": note}


def run_small_only(args):
    """Profiling aid: the acceptance kernels (`--only accept`) or SiLU-and-Mul (`--only silu`) at the
    step's shapes, a few hundred MB on the device, timed per call with CUDA events."""
    import vllm_rlt_b200 as rlt

    torch.cuda.set_device(0)
    device = torch.device("cuda", 0)
    work = Workload(seed=1234, requests=args.requests, layers=1)
    out = {"only": args.only, "requests": args.requests}

    def timed(fn):
        for _ in range(args.warmup):
            fn()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        for _ in range(args.steps):
            fn()
        b.record()
        torch.cuda.synchronize()
        return a.elapsed_time(b) / args.steps

    if args.only == "silu":
        out.update(silu_comparison(device, args.steps, args.warmup))
    else:
        x = {k: v.to(device) for k, v in work.host_inputs(pin=False).items() if k not in ("q", "k", "v", "gate", "up")}
        per_row_t = x["temperature"].repeat_interleave(TOKENS)
        slot_values = torch.zeros(2 * work.requests, 2, dtype=torch.int64, device=device)
        drafts, _ = rlt.sample_rows(x["draft"], per_row_t, x["u_draft"])
        tokens = torch.zeros(work.requests, TOKENS, dtype=torch.int64, device=device)
        tokens[:, 1:] = drafts.view(work.requests, TOKENS)[:, :-1]
        logits_bytes = x["target"].numel() * 4
        out["sample_rows_ms"] = timed(lambda: rlt.sample_rows(x["draft"], per_row_t, x["u_draft"]))
        out["accept_greedy_ms"] = timed(lambda: rlt.accept_greedy(x["target"], x["cu_rows"], tokens, x["starts"],
                                                                  x["slots"], slot_values))
        out["accept_rejection_ms"] = timed(lambda: rlt.accept_rejection(
            x["target"], x["draft"], x["cu_rows"], tokens, x["starts"], x["temperature"], x["u_accept"],
            x["u_final"], x["slots"], slot_values))
        result, _ = rlt.accept_rejection(x["target"], x["draft"], x["cu_rows"], tokens, x["starts"],
                                         x["temperature"], x["u_accept"], x["u_final"])
        accepted = result[work.accept_rows:work.accept_rows + work.requests]
        out["rollback_ms"] = timed(lambda: rlt.rollback(x["starts"], accepted + 1, x["request_tables"], BLOCK))
        # the same draws and acceptance with top-k = 50 / top-p = 0.9 on every request (radix-select cut)
        n = work.requests
        top_k, top_p = torch.full((n,), 50, dtype=torch.int32, device=device), torch.full((n,), 0.9, device=device)
        row_k, row_p = top_k.repeat_interleave(TOKENS), top_p.repeat_interleave(TOKENS)
        out["sample_rows_top_k_top_p_ms"] = timed(lambda: rlt.sample_rows(x["draft"], per_row_t, x["u_draft"], row_k, row_p))
        out["accept_rejection_top_k_top_p_ms"] = timed(lambda: rlt.accept_rejection(
            x["target"], x["draft"], x["cu_rows"], tokens, x["starts"], x["temperature"], x["u_accept"], x["u_final"],
            top_k=top_k, top_p=top_p))
        out["probabilities_top_p_ms"] = timed(lambda: rlt.probabilities(x["target"], per_row_t, None, row_p))
        out.update(rows=work.accept_rows, vocab=VOCAB, greedy_bytes=logits_bytes, rejection_bytes=2 * logits_bytes,
                   greedy_gbs=logits_bytes / out["accept_greedy_ms"] / 1e6,
                   rejection_gbs=2 * logits_bytes / out["accept_rejection_ms"] / 1e6)
    print(json.dumps(out))


def run_decode_workload(args):
    """Secondary workload (`--workload decode`): self-speculative decoding of a random-init
    Ouro-1.4B-shaped model (24 layers, hidden 2048, 16 x 128 MHA, FFN 5632, vocab 49152, 4 loops, bf16)
    through `vllm_rlt_b200.SelfSpeculativeDecoder` — the bench line's workload run to completion, with the output length set by
    `--output-tokens`.  The GEMMs are cuBLAS; every recurrent loop is replayed from a CUDA graph per
    row bucket unless `--eager` is given.  The prefill and the graph captures are outside the timed region."""
    import vllm_rlt_b200 as rlt

    torch.cuda.set_device(0)
    device = torch.device("cuda", 0)
    config = rlt.LoopedLMConfig()
    model = rlt.LoopedLM(config, rlt.seeded_state_dict(config, 3, device=device), device, torch.bfloat16)
    g = torch.Generator().manual_seed(11)
    lengths = torch.randint(args.prompt_min, args.prompt_max + 1, (args.requests,), generator=g).tolist()
    prompts = [torch.randint(1, config.vocab_size, (n,), generator=g).tolist() for n in lengths]
    if args.shared_prefix > 0:   # every second request starts with one common prefix (a long-context mix with shared prefixes)
        common = torch.randint(1, config.vocab_size, (args.shared_prefix,), generator=g).tolist()
        prompts = [common[:len(p) - 1] + p[len(common[:len(p) - 1]):] if i % 2 else p for i, p in enumerate(prompts)]
    decoder = rlt.SelfSpeculativeDecoder(model, cuda_graphs=not args.eager, prefix_caching=args.prefix_caching,
                                         capture_sizes=sorted({args.requests, max(args.requests // 2, 1),
                                                               max(args.requests // 4, 1)}))
    clock = {}

    def start_clock():
        torch.cuda.synchronize()
        clock["start"] = time.perf_counter()

    torch.cuda.synchronize()
    clock["begin"] = time.perf_counter()
    tokens = decoder.generate(prompts, args.output_tokens, num_speculative_tokens=args.k, draft_loops=DRAFT_LOOPS,
                              target_loops=TARGET_LOOPS, temperature=args.temperature, seed=1, after_prefill=start_clock,
                              in_flight=args.in_flight)
    torch.cuda.synchronize()
    seconds = time.perf_counter() - clock["start"]
    stats = decoder.stats
    # HBM roofline of the decode loop: every recurrent pass streams the layer weights once and the
    # K/V of every active request's context once per layer; every LM-head call streams lm_head once
    # (counted per draft pass and per round).  Activations and logits are left out (a few percent).
    c = config
    layer_params = (c.hidden_size * (c.num_attention_heads + 2 * c.num_key_value_heads) * c.head_dim
                    + c.num_attention_heads * c.head_dim * c.hidden_size + 3 * c.hidden_size * c.intermediate_size)
    weight_bytes = 2.0 * c.num_hidden_layers * layer_params * stats.loop_passes
    kv_bytes = 2.0 * 2 * c.num_key_value_heads * c.head_dim * c.num_hidden_layers * stats.context_tokens_read
    head_calls = stats.rounds / max(args.requests, 1) * (args.k + 1)   # upper bound: k draft calls + 1 verify call per round
    head_bytes = 2.0 * c.vocab_size * c.hidden_size * head_calls
    peak, peak_kind = measured_peaks()
    roofline_s = (weight_bytes + kv_bytes + head_bytes) / (peak * 1e9)
    print(json.dumps({
        "workload": f"decode: Ouro-1.4B-shaped random-init bf16, self-spec k={args.k} from depth 2, "
                    f"{args.requests} requests, prompts U[{args.prompt_min},{args.prompt_max}]"
                    + (f" (every second one behind a common {args.shared_prefix}-token prefix, prefix reuse "
                       f"{'on' if args.prefix_caching else 'off'})" if args.shared_prefix else "")
                    + f", {args.output_tokens} output tokens, T={args.temperature}, "
                    + ("eager launches" if args.eager else "every round one CUDA graph") + f", {args.in_flight} round(s) in flight",
        "total_seconds": time.perf_counter() - clock["begin"],
        "prefill_and_capture_seconds": clock["start"] - clock["begin"], "prompt_tokens": sum(lengths),
        "prompt_tokens_computed": stats.prompt_tokens_computed, "prefix_hit_tokens": stats.prefix_hit_tokens,
        "decode_seconds": seconds, "committed_tokens": stats.committed_tokens, "accepted_tokens": stats.accepted_tokens,
        "drafted_tokens": stats.drafted_tokens, "request_rounds": stats.rounds,
        "committed_tokens_per_s": stats.committed_tokens / seconds,
        "accepted_tokens_per_s": stats.accepted_tokens / seconds,
        "acceptance_rate": stats.accepted_tokens / max(stats.drafted_tokens, 1),
        "loop_passes": stats.loop_passes,
        "hbm_roofline": {"kv_bytes": kv_bytes, "weight_bytes": weight_bytes, "lm_head_bytes": head_bytes,
                         "peak_gbs": peak, "peak_kind": peak_kind, "seconds_at_peak": roofline_s,
                         "frac": roofline_s / seconds},
        "tokens_out": sum(len(t) for t in tokens), "attention_status": model.attention.last_status(device)}))


def run_reference_engine_workload(args):
    """`--workload decode --engine reference`: the decode workload's requests through the unmodified vllm-rlt
    engine on the GPU (an installed copy under baseline/_ref; nothing of this library on the path): the model
    class of the reference with the same seeded weights, its scheduler and speculative runner, its Triton paged
    attention, its CUDA graphs.  Timing follows the reference's own benchmark: the decode clock starts when
    every request has its first token and the device is idle, counts the tokens produced from then on and
    stops after the device has finished."""
    import vllm_rlt_b200 as rlt

    reference_root = ROOT / "baseline" / "_ref"
    if not (reference_root / "vllm_rlt").is_dir():
        print(json.dumps({"engine": "reference", "unavailable": "no copy of the reference under baseline/_ref"}))
        return
    sys.path.insert(0, str(reference_root))
    from vllm_rlt import CacheConfig, ExecutionConfig, SamplingParams, SpeculativeConfig
    from vllm_rlt.config import SchedulerConfig
    from vllm_rlt.engine.stage_engine import StageEngine
    from vllm_rlt.models import OuroConfig, OuroForCausalLM

    torch.cuda.set_device(0)
    device = torch.device("cuda", 0)
    ours = rlt.LoopedLMConfig()
    shape = {name: getattr(ours, name) for name in (
        "vocab_size", "hidden_size", "intermediate_size", "num_hidden_layers", "num_attention_heads",
        "num_key_value_heads", "head_dim", "rms_norm_eps", "rope_theta", "total_ut_steps")}
    config = OuroConfig(**shape, max_position_embeddings=4096, bos_token_id=0, eos_token_id=0)
    with torch.device(device):
        model = OuroForCausalLM(config).to(torch.bfloat16)
    state = rlt.seeded_state_dict(ours, 3, device=device)
    model.load_state_dict({name: state[name] for name in model.state_dict()}, strict=True)
    del state
    prompts = decode_prompts(args.requests, (args.prompt_min, args.prompt_max), config.vocab_size)
    pages = sum(-(-(len(p) + args.output_tokens + args.k + 2) // BLOCK) for p in prompts) * config.total_ut_steps + 64
    if args.adopt != "nothing":
        # What a maintainer of the reference adds to adopt the kernels: one more backend name that wraps
        # B200PagedAttention in the reference's own AttentionBackend / BackendCapabilities classes.
        import dataclasses

        from vllm_rlt.attention import backend as backend_module
        from vllm_rlt.core import kv_cache_manager as cache_module

        validate, create = backend_module.validate_backend_name, backend_module._create_explicit

        def explicit(name, device_, dtype, head_dim, block_size):
            if name != "b200":
                return create(name, device_, dtype, head_dim, block_size)
            native = rlt.create_backend(device_, dtype, head_dim, block_size)
            capabilities = backend_module.BackendCapabilities(**dataclasses.asdict(native.capabilities))
            return backend_module.AttentionBackend(native.kernel, capabilities, {"backend": "b200"})

        backend_module.validate_backend_name = cache_module.validate_backend_name = \
            lambda name: None if name == "b200" else validate(name)
        backend_module._create_explicit = explicit
        rlt.register_torch_op("vllm_rlt")
    engine = StageEngine(
        model, cache_config=CacheConfig(pages, BLOCK), attention_backend="triton" if args.adopt == "nothing" else "b200",
        scheduler_config=SchedulerConfig(max_num_seqs=args.requests,
                                         max_num_batched_tokens=max(2048, args.requests * (args.k + 1))),
        execution_config=ExecutionConfig(async_scheduling=not args.sync, cuda_graphs=not args.eager),
        speculative_config=SpeculativeConfig(args.k, draft_loops=DRAFT_LOOPS, target_loops=TARGET_LOOPS))
    if args.adopt == "runner":
        # ... and the runner: this library's looped LM over the reference's weights and KV-cache manager, in the place of
        # the engine's own speculative runner (device-resident protocol under the async engine, synchronous otherwise).
        native_model = rlt.LoopedLM(ours, model.state_dict(), device, torch.bfloat16)
        view = rlt.KVCacheManagerView(engine.cache_manager, max_pages=-(-config.max_position_embeddings // BLOCK))
        runner = rlt.B200SpeculativeRunner(
            native_model, view, rlt.SpeculativeConfig(args.k, draft_loops=DRAFT_LOOPS, target_loops=TARGET_LOOPS),
            max_num_seqs=args.requests, cuda_graphs=not args.eager, capture_sizes=[args.requests],
            compute_stream=engine.model_runner.core_stream, report_frontiers=not args.sync)
        engine.speculative_runner = engine.executor.speculation = runner
    params = SamplingParams(max_tokens=args.output_tokens, ignore_eos=True, temperature=args.temperature, seed=1)
    torch.cuda.synchronize()
    begin = time.perf_counter()
    for i, prompt in enumerate(prompts):
        engine.add_request(str(i), prompt, params)
    produced, finished, start, at_start = {}, 0, None, 0
    while engine.has_unfinished_requests():
        for output in engine.step():
            produced[output.request_id] = len(output.token_ids)
            finished += bool(output.finished)
        if start is None and len(produced) == args.requests:
            torch.cuda.synchronize()
            start, at_start = time.perf_counter(), sum(produced.values())
    torch.cuda.synchronize()
    seconds = time.perf_counter() - start
    stats = engine.speculative_runner.stats
    print(json.dumps({
        "engine": "vllm-rlt reference on the GPU, " + {"nothing": "unmodified", "attention": "with this library's attention "
                  "backend and SiLU op", "runner": "with this library's attention backend and speculative runner"}[args.adopt],
        "attention_backend": "triton" if args.adopt == "nothing" else "b200",
        "async_scheduling": not args.sync, "cuda_graphs": not args.eager,
        "workload": f"decode: Ouro-1.4B-shaped random-init bf16, self-spec k={args.k} from depth 2, {args.requests} requests, "
                    f"prompts U[{args.prompt_min},{args.prompt_max}], {args.output_tokens} output tokens, T={args.temperature}",
        "total_seconds": time.perf_counter() - begin, "prompt_pass_seconds": start - begin, "decode_seconds": seconds,
        "decode_tokens": sum(produced.values()) - at_start,
        "decode_tokens_per_s": (sum(produced.values()) - at_start) / seconds,
        "accepted_tokens": stats.accepted_tokens, "drafted_tokens": stats.drafted_tokens, "request_rounds": stats.rounds,
        "accepted_tokens_per_s_over_the_whole_run": stats.accepted_tokens / (time.perf_counter() - begin),
        "finished_requests": finished}))


# Layer shapes of the hybrid workload: width, attention (heads, kv heads), feed-forward width of the two-matrix MLP (and of
# the looped model's three-matrix one: the same parameters), Mamba-2 (heads, head size, state, groups), layers, vocabulary.
HYBRID_SIZES = {
    "2048": dict(width=2048, heads=16, kv_heads=16, ff=8448, looped_ff=5632, mamba=(64, 64, 128, 1), layers=12, vocab=49152),
    "4096": dict(width=4096, heads=32, kv_heads=8, ff=14336, looped_ff=9600, mamba=(128, 64, 128, 8), layers=8, vocab=49152),
}


def hybrid_config(size, pattern: str):
    """config.json of a Sobipel model whose layers repeat `pattern` ('a' attention, 'm' Mamba-2)."""
    heads, vdim, state, groups = size["mamba"]
    kinds = {"a": {"type": "attention", "mixer": {"heads": size["heads"], "kv_heads": size["kv_heads"], "dim": HEAD_DIM, "vdim": HEAD_DIM,
                                                  "scale": HEAD_DIM ** -0.5, "q_temp": {"coef": 0.1, "every": 2048}}},
             "m": {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": 4,
                                               "norm_groups": groups}}}
    layers = [dict(kinds[pattern[i % len(pattern)]], mlp={"kind": "dense", "ff": size["ff"]}) for i in range(size["layers"])]
    return {"architecture": "Sobipel", "vocab": size["vocab"], "width": size["width"], "norm": {"eps": 1e-6}, "layers": layers}


def device_weights(shapes, device, seed=0):
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in shapes.items():
        w = torch.randn(shape, device=device, generator=g) * (0.02 if len(shape) == 2 else 0.1)
        if "layernorm" in name or name in ("model.norm.weight",) or name.endswith("mix.norm"):
            w = w + 1
        out[name] = w.to(torch.bfloat16)
    return out


def timed_ms(run, steps: int, warmup: int) -> float:
    for _ in range(warmup):
        run()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    a.record()
    for _ in range(steps):
        run()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / steps


@torch.no_grad()
def hybrid_model_rows(name, model, steps, warmup):
    """Prefill and decode of one model through the engine: device time of a step, weights and caches larger than L2."""
    import vllm_rlt_b200 as rlt

    rows = []
    for requests, tokens in ((8, 2048), (1, 16384)):
        engine = rlt.Engine(model, max_tokens=requests * (tokens + 4 * BLOCK), max_sequences=requests, cuda_graphs=False)
        entries = [rlt.StepEntry(i, torch.randint(0, model.vocab_size, (tokens,)).tolist(), [tokens - 1]) for i in range(requests)]
        engine._claim(entries)
        batch = engine._batch(entries)
        last = batch.cu[1:].long() - 1
        ms = timed_ms(lambda: model.step_logits(model.forward_step(batch, engine.cache), last), steps, warmup)
        rows.append({"model": name, "phase": "prefill", "requests": requests, "tokens": tokens, "ms": ms, "tokens_per_s": requests * tokens / ms * 1e3})
        del engine, batch
    for requests, context in ((1, 4096), (16, 4096), (64, 2048)):
        engine = rlt.Engine(model, max_tokens=requests * (context + 4 * BLOCK), max_sequences=requests, max_sequence_tokens=context + BLOCK,
                            capture_sizes=[requests])
        for i in range(requests):
            engine.step([rlt.StepEntry(i, torch.randint(0, model.vocab_size, (context,)).tolist())])
        engine.step([rlt.StepEntry(i, [1], [0]) for i in range(requests)])
        (graph, *_), = engine._graphs.values()
        ms = timed_ms(graph.replay, steps * 4, warmup)
        rows.append({"model": name, "phase": "decode", "requests": requests, "tokens": context, "ms": ms, "tokens_per_s": requests / ms * 1e3})
        del engine, graph
    torch.cuda.empty_cache()
    return rows


def ring_us(calls, replays: int) -> float:
    """Microseconds per call of a ring of calls whose tensors together exceed L2, replayed from a CUDA graph."""
    for call in calls:
        call()
    torch.cuda.synchronize()
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        kept = [call() for call in calls]
    ms = timed_ms(graph.replay, replays, 2)
    del kept
    return ms / len(calls) * 1e3


class KernelRows:
    """Rows of a kernel table: time of a call in a ring of calls, and its fraction of the measured roofline (the later of the two bounds)."""

    def __init__(self, steps):
        self.steps, self.rows = steps, []
        self.peak_gbs, _ = measured_peaks()
        peaks = json.loads((ROOT / "MEASURED_PEAKS.json").read_text()) if (ROOT / "MEASURED_PEAKS.json").exists() else {}
        self.peak_tflops = float(peaks.get("bf16_tflops", 1590.0))

    def __call__(self, kernel, phase, like, make, nbytes=0.0, flops=0.0, copies=None):
        """make(i) -> a call on the i-th set of tensors."""
        copies = copies or max(2, min(48, int(400e6 // max(nbytes, 1)) + 1))
        calls = [make(i) for i in range(copies)]
        torch.cuda.synchronize()
        time.sleep(0.25)       # a row is timed in isolation, like the peaks: the clock has come back from the row before it
        us = ring_us(calls, self.steps)
        tensor = flops / self.peak_tflops / 1e6 > nbytes / self.peak_gbs / 1e3
        frac = flops / us / 1e6 / self.peak_tflops if tensor else nbytes / us / 1e3 / self.peak_gbs
        self.rows.append({"kernel": kernel, "phase": phase, "like": like, "us": us, "bound": "tensor" if tensor else "hbm", "roofline_frac": frac})
        torch.cuda.empty_cache()


@torch.no_grad()
def hybrid_kernel_rows(size, steps):
    """Every kernel of a hybrid layer at prefill (16384 rows: 8 x 2048) and decode (64 rows, context 2048), with its
    algorithmic bytes or flops against the measured peak, beside the like kernel of the looped model."""
    from types import SimpleNamespace

    import vllm_rlt_b200 as rlt

    device = torch.device("cuda", 0)
    peak_gbs, _ = measured_peaks()
    peaks = json.loads((ROOT / "MEASURED_PEAKS.json").read_text()) if (ROOT / "MEASURED_PEAKS.json").exists() else {}
    peak_tflops = float(peaks.get("bf16_tflops", 1590.0))
    width, heads, kv_heads, ff = size["width"], size["heads"], size["kv_heads"], size["ff"]
    m_heads, vdim, state, groups = size["mamba"]
    inner, gn = m_heads * vdim, groups * state
    channels = inner + 2 * gn
    bf16 = lambda *shape: torch.randn(*shape, device=device).to(torch.bfloat16)
    f32 = lambda *shape: torch.randn(*shape, device=device)
    rows_out = []

    def add(kernel, phase, like, make, nbytes=0.0, flops=0.0, copies=None):
        """make(i) -> a call on the i-th set of tensors."""
        copies = copies or max(2, min(48, int(400e6 // max(nbytes, 1)) + 1))
        us = ring_us([make(i) for i in range(copies)], steps)
        frac = flops / us / 1e6 / peak_tflops if flops else nbytes / us / 1e3 / peak_gbs
        rows_out.append({"kernel": kernel, "phase": phase, "like": like, "us": us, "bound": "tensor" if flops else "hbm",
                         "roofline_frac": frac})
        torch.cuda.empty_cache()

    for phase, seqs, new, context in (("prefill", 8, 2048, 2048), ("decode", 64, 1, 2048)):
        rows = seqs * new
        pages = context // BLOCK
        tables = torch.randperm(seqs * pages, device=device).int().view(seqs, pages)
        lengths = torch.full((seqs,), context, dtype=torch.int32, device=device)
        cu = (torch.arange(seqs + 1, device=device) * new).int()
        starts = lengths - new
        slots = torch.arange(seqs, device=device, dtype=torch.int32)
        row_seq = torch.arange(seqs, device=device, dtype=torch.int32).repeat_interleave(new)
        positions = (torch.arange(rows, device=device) % new).int() + (context - new)
        batch = SimpleNamespace(tables=tables[None], row_seq=row_seq, positions=positions)
        group = SimpleNamespace(sequences=seqs, max_new=new, cu=cu, starts=starts, slots=slots)
        terms = rlt.ScoreTerms(HEAD_DIM ** -0.5, 0.1, 2048, True)

        # attention: score terms against none, on the same cache
        kv_bytes = 2 * seqs * context * kv_heads * HEAD_DIM * 2
        qo_bytes = 2 * rows * heads * HEAD_DIM * 2
        visible = seqs * sum(range(context - new + 1, context + 1))
        flops = 4.0 * HEAD_DIM * heads * visible if new > 16 else 0.0
        sets = 2
        pools = [bf16(2, seqs * pages, BLOCK, kv_heads, HEAD_DIM) for _ in range(sets)]
        proj_width = (heads + 2 * kv_heads) * HEAD_DIM + ff
        q_wide = [bf16(rows, proj_width) for _ in range(sets)]
        out_wide = bf16(rows, heads * HEAD_DIM + ff)
        kernels = rlt.B200PagedAttention()

        def scored(i):
            q = q_wide[i % sets][:, :heads * HEAD_DIM].view(rows, heads, HEAD_DIM)
            out = out_wide[:, :heads * HEAD_DIM].view(rows, heads, HEAD_DIM)
            return lambda: kernels.scored(q, out, pools[i % sets][0], pools[i % sets][1], tables, lengths, cu, new, terms)

        q_plain = [bf16(rows, heads, HEAD_DIM) for _ in range(sets)]
        plain = lambda i: (lambda: kernels.prefill(q_plain[i % sets], pools[i % sets][0], pools[i % sets][1], tables, lengths, cu, new))
        add("scored attention", phase, None, scored, kv_bytes + qo_bytes, flops, copies=4)
        add("attention of the looped model", phase, "scored attention", plain, kv_bytes + qo_bytes, flops, copies=4)
        del q_plain

        # the same bytes and flops in 64-wide heads: the shape-general tensor-core kernels
        narrow = [pool.view(2, seqs * pages, BLOCK, 2 * kv_heads, HEAD_DIM // 2) for pool in pools]

        def scored_narrow(i):
            q = q_wide[i % sets][:, :heads * HEAD_DIM].view(rows, 2 * heads, HEAD_DIM // 2)
            out = out_wide[:, :heads * HEAD_DIM].view(rows, 2 * heads, HEAD_DIM // 2)
            return lambda: kernels.scored(q, out, narrow[i % sets][0], narrow[i % sets][1], tables, lengths, cu, new, terms)

        add("scored attention, 64-wide heads", phase, None, scored_narrow, kv_bytes + qo_bytes, flops, copies=4)
        del pools, narrow

        # the norm that opens a layer: 32-bit residual read and written, 16-bit contribution read, 16-bit row written
        copies = max(2, min(48, int(400e6 // (rows * width * 12)) + 1))
        res, delta, weight = [f32(rows, width) for _ in range(copies)], [bf16(rows, width) for _ in range(copies)], f32(width)
        add("residual_norm", phase, None, lambda i: (lambda: rlt.residual_norm(res[i], weight, 1e-6, torch.bfloat16, delta=delta[i], weight_offset=1.0)),
            rows * width * 12.0, copies=copies)
        res16, w16 = [bf16(rows, width) for _ in range(copies)], bf16(width)
        add("sandwich_norm", phase, "residual_norm",
            lambda i: (lambda: rlt.sandwich_norm(delta[i], w16, 1e-6, res16[i], w16, in_place=True)), rows * width * 8.0, copies=copies)
        del res, res16, delta

        # keys and values to their pages and gelu, against rope + KV write and silu-and-mul
        cache = bf16(2, seqs * pages, BLOCK, kv_heads, HEAD_DIM)
        kv_width = kv_heads * HEAD_DIM
        copies = max(2, min(48, int(400e6 // (rows * (2 * kv_width + ff) * 4)) + 1))
        projs = [bf16(rows, proj_width) for _ in range(copies)]
        add("block_epilogue", phase, None, lambda i: (lambda: rlt.block_epilogue(
            projs[i], batch, kv=(heads * HEAD_DIM, heads * HEAD_DIM + kv_width, cache[0], cache[1]),
            act=(heads * HEAD_DIM + 2 * kv_width, ff, "gelu", out_wide, heads * HEAD_DIM))), rows * (2 * kv_width + ff) * 4.0, copies=copies)
        cos = bf16(rows, HEAD_DIM)
        blocks = tables[row_seq.long(), (positions // BLOCK).long()].long()
        offsets = (positions % BLOCK).long()
        cut = lambda p, a, n: p[:, a * HEAD_DIM:(a + n) * HEAD_DIM].view(rows, n, HEAD_DIM)
        add("rope_kv_write", phase, "block_epilogue", lambda i: (lambda: rlt.rope_kv_write(
            cut(projs[i], 0, heads), cut(projs[i], heads, kv_heads), cut(projs[i], heads + kv_heads, kv_heads), cos, cos, cache[0], cache[1],
            blocks, offsets)), rows * ((heads + 2 * kv_heads) * HEAD_DIM * 4.0 + HEAD_DIM * 4), copies=copies)
        gate_up = [bf16(rows, 2 * size["looped_ff"]) for _ in range(copies)]
        add("silu_and_mul", phase, "block_epilogue", lambda i: (lambda: rlt.silu_and_mul_packed(gate_up[i])), rows * size["looped_ff"] * 6.0, copies=copies)
        del projs, gate_up, cache, q_wide, out_wide

        # the recurrent layer
        in_width = inner + channels + m_heads + ff
        conv_bytes = rows * (channels + ff) * 4.0
        copies = max(2, min(24, int(400e6 // conv_bytes) + 1))
        projs = [bf16(rows, in_width) for _ in range(copies)]
        mixed = [bf16(rows, channels) for _ in range(copies)]
        acted, y = bf16(rows, ff), bf16(rows, inner)
        conv_state = torch.zeros(seqs, 3, channels, device=device, dtype=torch.bfloat16)
        conv_w, conv_b = f32(channels, 4), f32(channels)
        add("causal_conv + gelu", phase, None, lambda i: (lambda: rlt.causal_conv(
            projs[i][:, inner:inner + channels], conv_w, conv_b, conv_state, mixed[i], group,
            act=(projs[i][:, inner + channels + m_heads:], "gelu", acted))), conv_bytes, copies=copies)
        dt_bias, a_log, d = f32(m_heads) - 3, f32(m_heads), f32(m_heads)
        ssm_sets = 2 if new > 1 else 4
        ssm = [torch.zeros(seqs, m_heads, state, vdim, device=device) for _ in range(ssm_sets)]

        def scan(i):
            x, b, c = mixed[i % copies].split((inner, gn, gn), 1)
            dt = projs[i % copies][:, inner + channels:inner + channels + m_heads]
            return lambda: rlt.ssd_scan(x, b, c, dt, dt_bias, a_log, d, ssm[i % ssm_sets], y, group)

        scan_bytes = rows * (channels + inner + m_heads) * 2.0 + 2 * ssm[0].numel() * 4.0
        add("ssd_scan", phase, None, scan, scan_bytes, copies=4)
        norm_w = f32(inner)
        outs = bf16(rows, inner + ff)
        add("gated_norm", phase, "sandwich_norm", lambda i: (lambda: rlt.gated_norm(
            y, projs[i][:, :inner], norm_w, outs[:, :inner], groups, 1e-6)), rows * inner * 6.0, copies=copies)
        del projs, mixed, acted, y, ssm, outs
    return rows_out


def run_hybrid_workload(args):
    """`--workload hybrid`: one JSON line with throughput rows, kernel rows and the clocks under them."""
    import vllm_rlt_b200 as rlt
    from vllm_rlt_b200.hybrid_lm import parameter_shapes as hybrid_shapes
    from vllm_rlt_b200.looped_lm import parameter_shapes as looped_shapes

    torch.cuda.set_device(0)
    device = torch.device("cuda", 0)
    report = {"workload": "hybrid", "data": "synthetic, random weights", "dtype": "bf16", "steps": args.steps, "sizes": {}}
    with ClockSampler(0) as clocks:
        for name, size in HYBRID_SIZES.items():
            rows = []
            for label, pattern in (("Sobipel, attention layers", "a"), ("Sobipel, Mamba-2 layers", "m"), ("Sobipel, 1 attention : 3 Mamba-2", "ammm")):
                config = rlt.HybridLMConfig.from_json(hybrid_config(size, pattern))
                model = rlt.HybridLM(config, device_weights(hybrid_shapes(config), device), device)
                rows += hybrid_model_rows(label, model, args.steps, args.warmup)
                del model
            looped = rlt.LoopedLMConfig(vocab_size=size["vocab"], hidden_size=size["width"], intermediate_size=size["looped_ff"],
                                        num_hidden_layers=size["layers"], num_attention_heads=size["heads"],
                                        num_key_value_heads=size["kv_heads"], head_dim=HEAD_DIM, total_ut_steps=1)
            model = rlt.LoopedLM(looped, device_weights(looped_shapes(looped), device), device, torch.bfloat16)
            rows += hybrid_model_rows("looped model, one loop", model, args.steps, args.warmup)
            del model
            torch.cuda.empty_cache()
            report["sizes"][name] = {"shape": {k: v for k, v in size.items()}, "throughput": rows, "kernels": hybrid_kernel_rows(size, args.steps)}
            torch.cuda.empty_cache()
    report["clocks"] = clocks.summary()
    print(json.dumps(report))


# Layer shapes of the stream workload: a Sugosun layer has the parameters of a looped layer of the same width (of the experts, those
# that a token uses).
STREAM_SIZES = {
    "2048": dict(width=2048, heads=16, q_rank=1536, kv_rank=512, rot_dim=64, window=1024, streams=4, experts=64, top=8, expert_ff=1024,
                 ff=5632, layers=8, vocab=49152),
    "4096": dict(width=4096, heads=32, q_rank=1536, kv_rank=512, rot_dim=64, window=1024, streams=4, experts=32, top=4, expert_ff=3584,
                 ff=9600, layers=6, vocab=49152),
}


def stream_config(size, pattern):
    """config.json of a Sugosun model whose layers repeat `pattern`: pairs of a mixer ('a' latent attention, 'l' lightning) and a
    feed-forward ('d' dense, 'e' experts)."""
    heads = size["heads"]
    mixers = {"a": ("latent_attention", {"heads": heads, "dim": HEAD_DIM, "rot_dim": size["rot_dim"], "vdim": HEAD_DIM, "q_rank": size["q_rank"],
                                         "kv_rank": size["kv_rank"], "scale": (HEAD_DIM + size["rot_dim"]) ** -0.5,
                                         "mask": {"size": size["window"]}, "rot": {"base": 10000.0, "dims": size["rot_dim"]}}),
              "l": ("lightning", {"heads": heads, "dim": HEAD_DIM, "vdim": HEAD_DIM, "decay": [1 - 2.0 ** -(2 + 8 * h / heads) for h in range(heads)]})}
    feeds = {"d": {"kind": "dense", "ff": size["ff"], "limit": 7.0},
             "e": {"kind": "moe", "router": {"experts": size["experts"], "top": size["top"]}, "expert": {"ff": size["expert_ff"]}}}
    layers = []
    for i in range(size["layers"]):
        mixer, feed = pattern[i % len(pattern)]
        layers.append({"type": mixers[mixer][0], "mixer": mixers[mixer][1], "mlp": feeds[feed]})
    return {"architecture": "Sugosun", "vocab": size["vocab"], "width": size["width"], "streams": size["streams"], "norm": {"eps": 1e-6},
            "embedding": {"bigram": {"buckets": 65521, "mul_prev": 8191, "mul_cur": 131}}, "layers": layers}


@torch.no_grad()
def stream_kernel_rows(size, steps):
    """Every kernel of a Sugosun layer at prefill (16384 rows: 8 x 2048) and decode (64 rows, context 2048), with its algorithmic bytes
    or flops against the measured peak, beside the like kernel of the looped model."""
    from types import SimpleNamespace

    import vllm_rlt_b200 as rlt
    from vllm_rlt_b200.engine import KeyRanges

    device = torch.device("cuda", 0)
    width, heads, rank, rot, q_rank = size["width"], size["heads"], size["kv_rank"], size["rot_dim"], size["q_rank"]
    ff, experts, top, expert_ff, s_count = size["ff"], size["experts"], size["top"], size["expert_ff"], size["streams"]
    row_dim, inner, key_dim = rank + rot, heads * HEAD_DIM, HEAD_DIM + rot
    bf16 = lambda *shape: torch.randn(*shape, device=device).to(torch.bfloat16)
    f32 = lambda *shape: torch.randn(*shape, device=device)
    add = KernelRows(steps)
    for phase, seqs, new, context in (("prefill", 8, 2048, 2048), ("decode", 64, 1, 2048)):
        rows, page = seqs * new, 64
        pages = context // page
        tables = torch.randperm(seqs * pages, device=device).int().view(seqs, pages)
        lengths = torch.full((seqs,), context, dtype=torch.int32, device=device)
        cu = (torch.arange(seqs + 1, device=device) * new).int()
        positions = (torch.arange(rows, device=device) % new).int() + (context - new)
        row_seq = torch.arange(seqs, device=device, dtype=torch.int32).repeat_interleave(new)
        batch = SimpleNamespace(tables=tables[None], row_seq=row_seq, positions=positions)
        group = SimpleNamespace(sequences=seqs, max_new=new, cu=cu, starts=lengths - new, slots=torch.arange(seqs, device=device, dtype=torch.int32))
        kernels = rlt.B200PagedAttention()
        small = lambda nbytes: max(2, min(48, int(400e6 // nbytes) + 1))

        # attention: pairs that are scored, with and without the window, and the looped model's of the same head count
        for window in (0, size["window"]):
            seen = [min(p + 1, window or context) for p in range(context - new, context)]
            name = f"latent attention, window {window}" if window else "latent attention, all keys"
            if new > 1:
                ranges = KeyRanges.of([(0, new)] * seqs, window, device)
                q, kv, latent, out = [bf16(rows, heads, key_dim) for _ in range(2)], [bf16(rows, 2 * inner) for _ in range(2)], bf16(rows, row_dim), bf16(rows, heads, HEAD_DIM)
                add(name, phase, "attention of the looped model",
                    lambda i: (lambda: rlt.latent_prompt_attention(q[i % 2], kv[i % 2], latent[:, rank:], out, HEAD_DIM, ranges, key_dim ** -0.5, window)),
                    rows * (heads * key_dim + 3 * inner + row_dim) * 2.0, 2.0 * sum(seen) * seqs * heads * (key_dim + HEAD_DIM), copies=4)
                del q, kv, latent, out
            else:
                copies = small(seqs * seen[0] * row_dim * 2)
                pools = [bf16(seqs * pages, page, 1, row_dim) for _ in range(copies)]
                q, out = bf16(rows, heads, row_dim), bf16(rows, heads, rank)
                add(name, phase, "attention of the looped model",
                    lambda i: (lambda: kernels.scored(q, out, pools[i], pools[i][..., :rank], tables, lengths, cu, 1, rlt.ScoreTerms(key_dim ** -0.5, window=window))),
                    seqs * seen[0] * row_dim * 2.0 + rows * heads * (row_dim + rank) * 2.0, 2.0 * seqs * seen[0] * heads * (row_dim + rank), copies=copies)
                del pools
        small_pages = context // BLOCK
        looped_tables = torch.randperm(seqs * small_pages, device=device).int().view(seqs, small_pages)
        pools = [bf16(2, seqs * small_pages, BLOCK, heads, HEAD_DIM) for _ in range(2)]
        q = [bf16(rows, heads, HEAD_DIM) for _ in range(2)]
        pairs = sum(range(context - new + 1, context + 1)) * seqs
        add("attention of the looped model", phase, None,
            lambda i: (lambda: kernels.prefill(q[i % 2], pools[i % 2][0], pools[i % 2][1], looped_tables, lengths, cu, new)),
            seqs * context * heads * HEAD_DIM * 4.0 + rows * inner * 4.0, 4.0 * pairs * inner, copies=4)
        del pools, q

        # between the sublayers
        nbytes = rows * width * (s_count * 8.0 + 4)
        copies = small(nbytes)
        streams, delta = [f32(rows, s_count, width) for _ in range(copies)], [bf16(rows, width) for _ in range(copies)]
        out_c, mix, reads, weight = f32(s_count), 0.3 * f32(s_count, s_count), f32(s_count), f32(width)
        add("stream_mix", phase, "sandwich_norm", lambda i: (lambda: rlt.stream_mix(streams[i], weight, 1e-6, torch.bfloat16, delta=delta[i], ran=(out_c, mix), follows=reads)),
            nbytes, copies=copies)
        parts = bf16(rows * top, width)
        places, shares = torch.randperm(rows * top, device=device).int().view(rows, top), torch.rand(rows, top, device=device)
        add("stream_mix, weighted parts", phase, "sandwich_norm", lambda i: (lambda: rlt.stream_mix(
            streams[i], weight, 1e-6, torch.bfloat16, delta=parts, parts=(places, shares), ran=(out_c, mix), follows=reads)),
            nbytes + rows * width * 2.0 * (top - 1), copies=copies)
        w16, res16 = bf16(width), [bf16(rows, width) for _ in range(copies)]
        add("sandwich_norm", phase, None, lambda i: (lambda: rlt.sandwich_norm(delta[i], w16, 1e-6, res16[i], w16, in_place=True)), rows * width * 8.0, copies=copies)
        del streams, delta, parts, res16

        # latent rows
        down = q_rank + row_dim
        nbytes = rows * down * 4.0
        copies = small(nbytes)
        proj, cache = [bf16(rows, down) for _ in range(copies)], bf16(seqs * pages, page, 1, row_dim)
        frequencies = rlt.rotation_frequencies(10000.0, rot, device)
        q_norm, kv_norm = f32(q_rank), f32(rank)
        add("latent_write", phase, "rope_kv_write", lambda i: (lambda: rlt.latent_write(proj[i], 0, q_rank, q_norm, kv_norm, 1e-6, frequencies, cache, batch)),
            nbytes, copies=copies)
        nbytes = rows * heads * rot * 4.0
        copies = small(rows * heads * key_dim * 2)
        q = [bf16(rows, heads, key_dim) for _ in range(copies)]
        add("rotate_heads", phase, "rope_kv_write", lambda i: (lambda: rlt.rotate_heads(q[i][:, :, HEAD_DIM:], q[i][:, :, HEAD_DIM:], frequencies, positions)), nbytes, copies=copies)
        del proj, q
        if new > 1:
            ranges = KeyRanges.of([(0, new)] * seqs, size["window"], device)
            caches = [bf16(seqs * pages, page, 1, row_dim) for _ in range(12)]
            add("latent_gather", phase, "rope_kv_write", lambda i: (lambda: rlt.latent_gather(caches[i], tables, ranges)), ranges.rows * row_dim * 4.0, copies=12)
            del caches
        copies = small(rows * inner * 8)
        k_cache = bf16(2, seqs * small_pages, BLOCK, heads, HEAD_DIM)
        qkv = [bf16(rows, 3 * inner) for _ in range(copies)]
        cos = bf16(rows, HEAD_DIM)
        blocks, offsets = looped_tables[row_seq.long(), (positions // BLOCK).long()].long(), (positions % BLOCK).long()
        cut = lambda p, a: p[:, a * inner:(a + 1) * inner].view(rows, heads, HEAD_DIM)
        add("rope_kv_write", phase, None, lambda i: (lambda: rlt.rope_kv_write(cut(qkv[i], 0), cut(qkv[i], 1), cut(qkv[i], 2), cos, cos, k_cache[0], k_cache[1], blocks, offsets)),
            rows * (3 * inner * 4.0 + HEAD_DIM * 4), copies=copies)
        del k_cache, qkv

        # lightning attention
        copies = small(rows * inner * 8)
        proj = [bf16(rows, 4 * inner) for _ in range(copies)]
        mixed = [bf16(rows, 3 * inner) for _ in range(min(copies, 4))]
        add("block_epilogue (silu)", phase, "silu_and_mul", lambda i: (lambda: rlt.block_epilogue(proj[i], batch, act=(0, 3 * inner, "silu", mixed[i % len(mixed)], 0))),
            rows * 3 * inner * 4.0, copies=copies)
        y, table = bf16(rows, inner), rlt.decay_table([1 - 2.0 ** -(2 + 8 * h / heads) for h in range(heads)], device)
        states = [torch.zeros(seqs, heads, HEAD_DIM, HEAD_DIM, device=device) for _ in range(4)]
        add("decay_scan", phase, None, lambda i: (lambda: rlt.decay_scan(
            *(mixed[i % len(mixed)][:, a * inner:(a + 1) * inner] for a in range(3)), table, states[i % 4], y, group)),
            rows * 4 * inner * 2.0 + 2 * states[0].numel() * 4.0, copies=4)
        norm_w, gated = f32(inner), bf16(rows, inner)
        add("gated_norm (gate behind)", phase, "sandwich_norm", lambda i: (lambda: rlt.gated_norm(y, proj[i][:, 3 * inner:], norm_w, gated, 1, 1e-6, gate_behind=True)),
            rows * inner * 6.0, copies=copies)
        del proj, mixed, y, states, gated

        # feed-forwards
        copies = small(rows * ff * 6)
        gate_up = [bf16(rows, 2 * ff) for _ in range(copies)]
        add("clamped_glu", phase, "silu_and_mul", lambda i: (lambda: rlt.clamped_glu(gate_up[i], ff, ff, 7.0, 1.702)), rows * ff * 6.0, copies=copies)
        add("silu_and_mul", phase, None, lambda i: (lambda: rlt.silu_and_mul_packed(gate_up[i])), rows * ff * 6.0, copies=copies)
        del gate_up
        logits, correction = [f32(rows, experts) for _ in range(4)], 0.01 * f32(experts)
        routing = rlt.expert_route(logits[0], correction, top)
        add("expert_route (with its zeroing)", phase, "sandwich_norm", lambda i: (lambda: rlt.expert_route(logits[i % 4], correction, top)), rows * (experts * 4.0 + top * 12), copies=8)
        h = [bf16(rows, width) for _ in range(4)]
        add("expert_gather", phase, "rope_kv_write", lambda i: (lambda: rlt.expert_gather(h[i % 4], routing)), rows * (1 + top) * width * 2.0, copies=4)
        used = int((routing.counts > 0).sum())
        up, downs = [bf16(experts, expert_ff, width) for _ in range(2)], [bf16(experts, width, expert_ff) for _ in range(2)]
        x, act = rlt.expert_gather(h[0], routing), bf16(rows * top, expert_ff)
        nbytes, flops = used * width * expert_ff * 2.0 + rows * top * (width + expert_ff) * 2.0, 2.0 * rows * top * width * expert_ff
        add("expert_gemm, up and squared relu", phase, "cuBLAS GEMM", lambda i: (lambda: rlt.expert_gemm(x, up[i % 2], routing.counts, "squared_relu")), nbytes, flops, copies=4)
        add("expert_gemm, down", phase, "cuBLAS GEMM", lambda i: (lambda: rlt.expert_gemm(act, downs[i % 2], routing.counts)), nbytes, flops, copies=4)
        del up, downs, x, act, h
        dense, inputs = [bf16(2 * ff, width) for _ in range(8)], bf16(rows, width)
        add("cuBLAS GEMM (gate and up)", phase, None, lambda i: (lambda: torch.nn.functional.linear(inputs, dense[i])),
            (2 * ff * width + rows * (width + 2 * ff)) * 2.0, 2.0 * rows * width * 2 * ff, copies=8)
        del dense, inputs
    return add.rows


def run_stream_workload(args):
    """`--workload stream`: one JSON line with throughput rows, kernel rows and the clocks under them."""
    import vllm_rlt_b200 as rlt
    from vllm_rlt_b200.looped_lm import parameter_shapes as looped_shapes
    from vllm_rlt_b200.stream_lm import parameter_shapes as stream_shapes

    torch.cuda.set_device(0)
    device = torch.device("cuda", 0)
    report = {"workload": "stream", "data": "synthetic, random weights", "dtype": "bf16", "steps": args.steps, "sizes": {}}
    with ClockSampler(0) as clocks:
        for name, size in STREAM_SIZES.items():
            rows = []
            for label, pattern in (("Sugosun, latent attention and dense", ["ad"]), ("Sugosun, lightning and dense", ["ld"]),
                                   ("Sugosun, latent attention and experts", ["ae"]), ("Sugosun, 1 latent : 3 lightning, experts", ["ae", "le", "le", "le"])):
                config = rlt.StreamLMConfig.from_json(stream_config(size, pattern))
                model = rlt.StreamLM(config, device_weights(stream_shapes(config), device), device)
                rows += hybrid_model_rows(label, model, args.steps, args.warmup)
                del model
                torch.cuda.empty_cache()
            looped = rlt.LoopedLMConfig(vocab_size=size["vocab"], hidden_size=size["width"], intermediate_size=size["ff"],
                                        num_hidden_layers=size["layers"], num_attention_heads=size["heads"],
                                        num_key_value_heads=size["heads"], head_dim=HEAD_DIM, total_ut_steps=1)
            model = rlt.LoopedLM(looped, device_weights(looped_shapes(looped), device), device, torch.bfloat16)
            rows += hybrid_model_rows("looped model, one loop", model, args.steps, args.warmup)
            del model
            torch.cuda.empty_cache()
            report["sizes"][name] = {"shape": dict(size), "throughput": rows, "kernels": stream_kernel_rows(size, args.steps)}
            torch.cuda.empty_cache()
    report["clocks"] = clocks.summary()
    print(json.dumps(report))


# Layer shapes of the sandwich workload: those of the stream workload's latent and dense layers, with windowed attention of grouped heads.
SANDWICH_SIZES = {
    "2048": dict(width=2048, heads=16, kv_heads=4, q_rank=1536, kv_rank=512, rot_dim=64, window=1024, taps=4, ff=5632, layers=8, vocab=49152),
    "4096": dict(width=4096, heads=32, kv_heads=8, q_rank=1536, kv_rank=512, rot_dim=64, window=1024, taps=4, ff=9600, layers=6, vocab=49152),
}


def sandwich_config(size, pattern):
    """config.json of a Kezuvik model whose layers repeat `pattern` ('e' latent attention with a gate per element, 's' latent attention with
    sinks, scaled rotation and a gate per head, 'w' windowed attention)."""
    latent = {"heads": size["heads"], "dim": HEAD_DIM, "rot_dim": size["rot_dim"], "vdim": HEAD_DIM, "q_rank": size["q_rank"], "kv_rank": size["kv_rank"],
              "scale": (HEAD_DIM + size["rot_dim"]) ** -0.5}
    rot = {"base": 10000.0, "dims": size["rot_dim"]}
    kinds = {"e": ("latent_attention", dict(latent, rot=rot)),
             "s": ("latent_attention_2", dict(latent, rot=dict(rot, scaling={"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}))),
             "w": ("attention", {"heads": size["heads"], "kv_heads": size["kv_heads"], "dim": HEAD_DIM, "vdim": HEAD_DIM, "conv": size["taps"],
                                 "mask": {"size": size["window"]}, "scale": HEAD_DIM ** 0.5})}
    layers = []
    for i in range(size["layers"]):
        kind, mixer = kinds[pattern[i % len(pattern)]]
        layers.append({"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": size["ff"]}})
    return {"architecture": "Kezuvik", "vocab": size["vocab"], "width": size["width"], "residual_mult": 0.5, "logit_softcap": 30.0,
            "norm": {"eps": 1e-6}, "layers": layers}


@torch.no_grad()
def sandwich_kernel_rows(size, steps):
    """Every kernel of a Kezuvik layer at prefill (16384 rows: 8 x 2048) and decode (64 rows, context 2048), with its algorithmic bytes
    or flops against the measured peak, beside the like kernel of the nearest model (Sugosun, Sobipel, looped)."""
    from types import SimpleNamespace

    import vllm_rlt_b200 as rlt
    from vllm_rlt_b200.engine import KeyRanges

    device = torch.device("cuda", 0)
    width, heads, kv_heads, rank, rot, q_rank = (size[k] for k in ("width", "heads", "kv_heads", "kv_rank", "rot_dim", "q_rank"))
    ff, window, taps = size["ff"], size["window"], size["taps"]
    row_dim, inner, key_dim, kv_inner = rank + rot, heads * HEAD_DIM, HEAD_DIM + rot, kv_heads * HEAD_DIM
    bf16 = lambda *shape: torch.randn(*shape, device=device).to(torch.bfloat16)
    f32 = lambda *shape: torch.randn(*shape, device=device)
    add = KernelRows(steps)
    sink = f32(heads)
    for phase, seqs, new, context in (("prefill", 8, 2048, 2048), ("decode", 64, 1, 2048)):
        rows, page = seqs * new, 64
        pages = context // page
        tables = torch.randperm(seqs * pages, device=device).int().view(seqs, pages)
        lengths = torch.full((seqs,), context, dtype=torch.int32, device=device)
        cu = (torch.arange(seqs + 1, device=device) * new).int()
        positions = (torch.arange(rows, device=device) % new).int() + (context - new)
        row_seq = torch.arange(seqs, device=device, dtype=torch.int32).repeat_interleave(new)
        batch = SimpleNamespace(tables=tables[None], row_seq=row_seq, positions=positions)
        group = SimpleNamespace(sequences=seqs, max_new=new, cu=cu, starts=lengths - new, slots=torch.arange(seqs, device=device, dtype=torch.int32),
                                lengths=lengths, tables=tables)
        kernels = rlt.B200PagedAttention()
        small = lambda nbytes: max(2, min(48, int(400e6 // nbytes) + 1))

        # latent attention: sinks and gates against none
        pairs = sum(range(context - new + 1, context + 1)) * seqs
        if new > 1:
            ranges = KeyRanges.of([(0, new)] * seqs, 0, device)
            q, kv, latent, out = [bf16(rows, heads, key_dim) for _ in range(2)], [bf16(rows, 2 * inner) for _ in range(2)], bf16(rows, row_dim), bf16(rows, heads, HEAD_DIM)
            gates = {"head": bf16(rows, heads), "element": bf16(rows, inner)}
            for name, like, extra in (("latent attention, sink, gate per head", "latent attention (Sugosun)", dict(sink=sink, gate=gates["head"])),
                                      ("latent attention, gate per element", "latent attention (Sugosun)", dict(gate=gates["element"])),
                                      ("latent attention (Sugosun)", None, {})):
                nbytes = rows * (heads * key_dim + 3 * inner + row_dim) * 2.0 + (extra["gate"].numel() * 2.0 if extra else 0.0)
                add(name, phase, like, lambda i: (lambda: rlt.latent_prompt_attention(q[i % 2], kv[i % 2], latent[:, rank:], out, HEAD_DIM, ranges, key_dim ** -0.5, 0, **extra)),
                    nbytes, 2.0 * pairs * heads * (key_dim + HEAD_DIM), copies=4)
            del q, kv, latent, out, gates
        else:
            copies = small(seqs * context * row_dim * 2)
            pools = [bf16(seqs * pages, page, 1, row_dim) for _ in range(copies)]
            q, out = bf16(rows, heads, row_dim), bf16(rows, heads, rank)
            for name, like, terms in (("latent attention, sink", "latent attention (Sugosun)", rlt.ScoreTerms(key_dim ** -0.5, sink=sink)),
                                      ("latent attention (Sugosun)", None, rlt.ScoreTerms(key_dim ** -0.5))):
                add(name, phase, like, lambda i: (lambda: kernels.scored(q, out, pools[i], pools[i][..., :rank], tables, lengths, cu, 1, terms)),
                    seqs * context * row_dim * 2.0 + rows * heads * (row_dim + rank) * 2.0, 2.0 * seqs * context * heads * (row_dim + rank), copies=copies)
            del pools, q, out

        # windowed attention of grouped heads, and the page kernels' over whole contexts with the same heads
        seen = sum(min(p + 1, window) for p in range(context - new, context)) * seqs
        stored = seqs * min(context, new + window - 1)
        q, out = [bf16(rows, heads, HEAD_DIM) for _ in range(2)], bf16(rows, heads, HEAD_DIM)
        terms = rlt.ScoreTerms(HEAD_DIM ** -0.5, window=window)
        kv_bytes, qo_bytes = stored * kv_inner * 4.0, rows * inner * 4.0
        if new > 1:
            ranges = KeyRanges.of([(0, new)] * seqs, window, device)
            k, v, gate = bf16(ranges.rows, kv_heads, HEAD_DIM), bf16(ranges.rows, kv_heads, HEAD_DIM), bf16(rows, inner)
            add("windowed attention, gate per element", phase, "attention of grouped heads (Sobipel)",
                lambda i: (lambda: rlt.packed_attention(q[i % 2], k, v, out, ranges, HEAD_DIM ** -0.5, window, gate=gate)), kv_bytes + 1.5 * qo_bytes, 4.0 * seen * inner, copies=4)
            del k, v, gate
            caches = [bf16(seqs * pages, page, 1, kv_inner) for _ in range(12)]
            add("latent_gather (keys of a window)", phase, "latent_gather (Sugosun)", lambda i: (lambda: rlt.latent_gather(caches[i], tables, ranges)),
                ranges.rows * kv_inner * 4.0, copies=12)
            caches = [bf16(seqs * pages, page, 1, row_dim) for _ in range(12)]
            add("latent_gather (Sugosun)", phase, None, lambda i: (lambda: rlt.latent_gather(caches[i], tables, ranges)), ranges.rows * row_dim * 4.0, copies=12)
            del caches
        else:
            copies = small(kv_bytes)
            pools = [bf16(2, seqs * pages, page, kv_heads, HEAD_DIM) for _ in range(copies)]
            add("windowed attention", phase, "attention of grouped heads (Sobipel)",
                lambda i: (lambda: kernels.scored(q[i % 2], out, pools[i][0], pools[i][1], tables, lengths, cu, 1, terms)), kv_bytes + qo_bytes, copies=copies)
            del pools
        small_pages = context // BLOCK
        small_tables = torch.randperm(seqs * small_pages, device=device).int().view(seqs, small_pages)
        copies = max(2, min(12, small(seqs * context * kv_inner * 4)))
        pools = [bf16(2, seqs * small_pages, BLOCK, kv_heads, HEAD_DIM) for _ in range(copies)]
        plain = rlt.ScoreTerms(HEAD_DIM ** -0.5, 0.1, 2048, True)
        add("attention of grouped heads (Sobipel)", phase, None,
            lambda i: (lambda: kernels.scored(q[i % 2], out, pools[i][0], pools[i][1], small_tables, lengths, cu, new, plain)),
            seqs * context * kv_inner * 4.0 + qo_bytes, 4.0 * pairs * inner, copies=copies)
        del pools, q, out

        # between projections and scores
        channels = inner + 2 * kv_inner
        nbytes = rows * channels * 4.0 + (seqs * (taps - 1) * channels * 4.0 if new == 1 else 0.0)
        copies = small(rows * (channels + inner) * 2)
        proj = [bf16(rows, channels + inner) for _ in range(copies)]
        weight, state = f32(taps, channels), torch.zeros(seqs, taps - 1, channels, dtype=torch.bfloat16, device=device)
        q_out, cache = bf16(rows, heads, HEAD_DIM), bf16(2, seqs * pages, page, kv_heads, HEAD_DIM)
        add("conv_heads", phase, "causal_conv (Sobipel)",
            lambda i: (lambda: rlt.conv_heads(proj[i], (0, inner, inner + kv_inner), weight, 1e-6, state, q_out, cache[0], cache[1], group)), nbytes, copies=copies)
        channel_weight, bias, mixed = f32(channels, taps), f32(channels), bf16(rows, channels)
        add("causal_conv (Sobipel)", phase, None, lambda i: (lambda: rlt.causal_conv(proj[i][:, :channels], channel_weight, bias, state, mixed, group)), nbytes, copies=copies)
        del proj, q_out, cache, mixed
        nbytes = rows * heads * rot * 4.0
        copies = small(rows * heads * key_dim * 2)
        q = [bf16(rows, heads, key_dim) for _ in range(copies)]
        frequencies = rlt.rotation_frequencies(10000.0, rot, device)
        for name, like, turn in (("rotate_heads (halves)", "rotate_heads (Sugosun)", dict(halves=True, amplitude=1.2)), ("rotate_heads (Sugosun)", None, {})):
            add(name, phase, like, lambda i: (lambda: rlt.rotate_heads(q[i][:, :, HEAD_DIM:], q[i][:, :, HEAD_DIM:], frequencies, positions, **turn)), nbytes, copies=copies)
        del q
        down = q_rank + row_dim
        copies = small(rows * down * 4)
        proj, cache = [bf16(rows, down) for _ in range(copies)], bf16(seqs * pages, page, 1, row_dim)
        q_norm, kv_norm = f32(q_rank), f32(rank)
        for name, like, turn in (("latent_write (halves)", "latent_write (Sugosun)", dict(halves=True, amplitude=1.2)), ("latent_write (Sugosun)", None, {})):
            add(name, phase, like, lambda i: (lambda: rlt.latent_write(proj[i], 0, q_rank, q_norm, kv_norm, 1e-6, frequencies, cache, batch, **turn)), rows * down * 4.0, copies=copies)
        del proj, cache

        # between the sublayers
        nbytes = rows * width * 12.0
        copies = small(nbytes)
        residual, delta = [f32(rows, width) for _ in range(copies)], [bf16(rows, width) for _ in range(copies)]
        before, behind = f32(width), f32(width)
        add("residual_norm, layer norms on both sides", phase, "sandwich_norm (looped)",
            lambda i: (lambda: rlt.residual_norm(residual[i], before, 1e-6, torch.bfloat16, delta=delta[i], behind=(behind, 0.5), centred=True)), nbytes, copies=copies)
        add("residual_norm (Sobipel)", phase, None, lambda i: (lambda: rlt.residual_norm(residual[i], before, 1e-6, torch.bfloat16, delta=delta[i])), nbytes, copies=copies)
        w16, res16 = bf16(width), [bf16(rows, width) for _ in range(copies)]
        add("sandwich_norm (looped)", phase, None, lambda i: (lambda: rlt.sandwich_norm(delta[i], w16, 1e-6, res16[i], w16, in_place=True)), rows * width * 8.0, copies=copies)
        del residual, delta, res16

        # gates and units
        copies = small(rows * inner * 4)
        y, gate = [bf16(rows, heads, HEAD_DIM) for _ in range(copies)], [bf16(rows, inner) for _ in range(copies)]
        add("head_gate, per element", phase, "gated_norm (Sugosun)", lambda i: (lambda: rlt.head_gate(y[i], gate[i])), rows * inner * 6.0, copies=copies)
        add("head_gate, per head", phase, "gated_norm (Sugosun)", lambda i: (lambda: rlt.head_gate(y[i], gate[i][:, :heads])), rows * inner * 4.0, copies=copies)
        norm_w, gated = f32(inner), bf16(rows, inner)
        add("gated_norm (Sugosun)", phase, None, lambda i: (lambda: rlt.gated_norm(y[i].view(rows, -1), gate[i], norm_w, gated, 1, 1e-6, gate_behind=True)), rows * inner * 6.0, copies=copies)
        del y, gate, gated
        copies = small(rows * ff * 6)
        gate_up = [bf16(rows, 2 * ff) for _ in range(copies)]
        add("gated_unit (tanh gelu)", phase, "clamped_glu (Sugosun)", lambda i: (lambda: rlt.gated_unit(gate_up[i], ff, ff, "gelu_tanh")), rows * ff * 6.0, copies=copies)
        add("clamped_glu (Sugosun)", phase, None, lambda i: (lambda: rlt.clamped_glu(gate_up[i], ff, ff, 7.0, 1.702)), rows * ff * 6.0, copies=copies)
        del gate_up
        if new == 1:
            copies = small(rows * size["vocab"] * 4)
            logits = [f32(rows, size["vocab"]) for _ in range(copies)]
            add("soft_cap", phase, "gated_norm (Sugosun)", lambda i: (lambda: rlt.soft_cap(logits[i], 30.0)), rows * size["vocab"] * 8.0, copies=copies)
            del logits
    return add.rows


def run_sandwich_workload(args):
    """`--workload sandwich`: one JSON line with throughput rows, kernel rows and the clocks under them."""
    import vllm_rlt_b200 as rlt
    from vllm_rlt_b200.looped_lm import parameter_shapes as looped_shapes
    from vllm_rlt_b200.sandwich_lm import parameter_shapes as sandwich_shapes
    from vllm_rlt_b200.stream_lm import parameter_shapes as stream_shapes

    torch.cuda.set_device(0)
    device = torch.device("cuda", 0)
    report = {"workload": "sandwich", "data": "synthetic, random weights", "dtype": "bf16", "steps": args.steps, "sizes": {}}
    with ClockSampler(0) as clocks:
        for name, size in SANDWICH_SIZES.items():
            rows = []
            builds = [(f"Kezuvik, {label}", lambda pattern=pattern: rlt.SandwichLM(config := rlt.SandwichLMConfig.from_json(sandwich_config(size, pattern)),
                                                                                   device_weights(sandwich_shapes(config), device), device))
                      for label, pattern in (("latent attention, gate per element", "e"), ("latent attention, sinks", "s"), ("windowed attention", "w"),
                                             ("all three", "sew"))]
            builds.append(("Sugosun, latent attention and dense", lambda: rlt.StreamLM(
                config := rlt.StreamLMConfig.from_json(stream_config(STREAM_SIZES[name], ["ad"])), device_weights(stream_shapes(config), device), device)))
            looped = rlt.LoopedLMConfig(vocab_size=size["vocab"], hidden_size=size["width"], intermediate_size=size["ff"],
                                        num_hidden_layers=size["layers"], num_attention_heads=size["heads"],
                                        num_key_value_heads=size["heads"], head_dim=HEAD_DIM, total_ut_steps=1)
            builds.append(("looped model, one loop", lambda: rlt.LoopedLM(looped, device_weights(looped_shapes(looped), device), device, torch.bfloat16)))
            for label, build in builds:
                model = build()
                rows += hybrid_model_rows(label, model, args.steps, args.warmup)
                del model
                torch.cuda.empty_cache()
            report["sizes"][name] = {"shape": dict(size), "throughput": rows, "kernels": sandwich_kernel_rows(size, args.steps)}
            torch.cuda.empty_cache()
    report["clocks"] = clocks.summary()
    print(json.dumps(report))


# Layer shapes of the postnorm workload: the windowed attention of the sandwich workload, recurrent layers with heads of the same size, and the
# dense and mixture-of-experts feed-forwards of the stream workload.
POSTNORM_SIZES = {
    "2048": dict(width=2048, heads=16, kv_heads=4, rank=128, window=1024, keep=4, taps=4, ff=5632, experts=64, top=8, expert_ff=704, layers=8, vocab=49152),
    "4096": dict(width=4096, heads=32, kv_heads=8, rank=128, window=1024, keep=4, taps=4, ff=9600, experts=32, top=4, expert_ff=2400, layers=6, vocab=49152),
}


def postnorm_config(size, pattern):
    """config.json of a Degavik model whose layers repeat `pattern`: pairs of a mixer ('c' gated delta rule, 'r' retention, 't' talking attention)
    and a feed-forward ('d' dense, 'e' experts with a shared one)."""
    heads = size["heads"]
    rot = {"base": 10000.0, "dims": HEAD_DIM}
    mixers = {"c": ("channel_delta", {"heads": heads, "kv_heads": heads, "dim": HEAD_DIM, "vdim": HEAD_DIM, "conv": size["taps"]}),
              "r": ("retention", {"heads": heads, "dim": HEAD_DIM, "vdim": HEAD_DIM, "rot": rot, "decay": [1 - 2.0 ** -(2 + 8 * h / heads) for h in range(heads)]}),
              "t": ("attention", {"heads": heads, "kv_heads": size["kv_heads"], "dim": HEAD_DIM, "vdim": HEAD_DIM, "scale": HEAD_DIM ** -0.5, "softcap": 20.0,
                                  "rot": dict(rot, dims=HEAD_DIM // 2), "mask": {"size": size["window"], "keep_first": size["keep"]}})}
    feeds = {"d": {"kind": "dense", "ff": size["ff"]},
             "e": {"kind": "moe", "router": {"experts": size["experts"], "top": size["top"]}, "expert": {"ff": size["expert_ff"]}, "shared": {"ff": size["expert_ff"]}}}
    layers = []
    for i in range(size["layers"]):
        mixer, feed = pattern[i % len(pattern)]
        layers.append({"type": mixers[mixer][0], "mixer": mixers[mixer][1], "mlp": feeds[feed]})
    return {"architecture": "Degavik", "vocab": size["vocab"], "width": size["width"], "norm": {"eps": 1e-6}, "layers": layers}


@torch.no_grad()
def postnorm_kernel_rows(size, steps):
    """Every kernel of a Degavik layer at prefill (16384 rows: 8 x 2048) and decode (64 rows, context 2048), with its algorithmic bytes
    or flops against the measured peak, beside the like kernel of the nearest model (Kezuvik, Sugosun, Sobipel).  Talking attention's flops are
    those of mixing the weights first: two products and a heads x heads matrix per pair."""
    from types import SimpleNamespace

    import vllm_rlt_b200 as rlt
    from vllm_rlt_b200.engine import KeyRanges

    device = torch.device("cuda", 0)
    width, heads, kv_heads, rank, ff = (size[k] for k in ("width", "heads", "kv_heads", "rank", "ff"))
    window, keep, taps, experts, top, expert_ff = (size[k] for k in ("window", "keep", "taps", "experts", "top", "expert_ff"))
    inner, kv_inner = heads * HEAD_DIM, kv_heads * HEAD_DIM
    bf16 = lambda *shape: torch.randn(*shape, device=device).to(torch.bfloat16)
    f32 = lambda *shape: torch.randn(*shape, device=device)
    add = KernelRows(steps)
    terms = rlt.ScoreTerms(HEAD_DIM ** -0.5, window=window, keep_first=keep, softcap=20.0, head_scale=1 + 0.1 * f32(heads))
    talk = torch.eye(heads, device=device) + 0.1 * f32(heads, heads)
    for phase, seqs, new, context in (("prefill", 8, 2048, 2048), ("decode", 64, 1, 2048)):
        rows, page = seqs * new, 64
        pages = context // page
        tables = torch.randperm(seqs * pages, device=device).int().view(seqs, pages)
        lengths = torch.full((seqs,), context, dtype=torch.int32, device=device)
        cu = (torch.arange(seqs + 1, device=device) * new).int()
        positions = (torch.arange(rows, device=device) % new).int() + (context - new)
        row_seq = torch.arange(seqs, device=device, dtype=torch.int32).repeat_interleave(new)
        batch = SimpleNamespace(tables=tables[None], row_seq=row_seq, positions=positions)
        group = SimpleNamespace(sequences=seqs, max_new=new, cu=cu, local_cu=cu, starts=lengths - new, slots=torch.arange(seqs, device=device, dtype=torch.int32),
                                lengths=lengths, tables=tables, portions=[(0, new)] * seqs if new > 1 else None)
        kernels = rlt.B200PagedAttention()
        small = lambda nbytes: max(2, min(48, int(400e6 // nbytes) + 1))

        # attention
        seen = sum(min(p + 1, window) + max(min(keep, p + 1 - window), 0) for p in range(context - new, context)) * seqs
        stored = seqs * min(context, new + window + keep - 1)
        q, out = [bf16(rows, heads, HEAD_DIM) for _ in range(2)], bf16(rows, heads, HEAD_DIM)
        kv_bytes, qo_bytes = stored * kv_inner * 4.0, rows * inner * 4.0
        if new > 1:
            ranges, plain_ranges = KeyRanges.of([(0, new)] * seqs, window, device, keep, 128), KeyRanges.of([(0, new)] * seqs, window, device)
            k, v, gate = bf16(ranges.rows, kv_inner), bf16(ranges.rows, kv_inner), bf16(rows, inner)
            spread = bf16(rows, heads, kv_inner)
            add("talking attention, spread output", phase, "windowed attention (Kezuvik)",
                lambda i: (lambda: rlt.talking_prompt(q[i % 2], k, v, spread, ranges, terms, kv_heads)), kv_bytes + qo_bytes, seen * heads * (4.0 * HEAD_DIM + 2 * heads), copies=4)
            add("head_mix", phase, "head_gate (Kezuvik)", lambda i: (lambda: rlt.head_mix(spread, talk, out, kv_heads)), rows * (heads * kv_inner + inner) * 2.0, copies=2)

            def whole(i):
                def call():
                    rlt.talking_prompt(q[i % 2], k, v, spread, ranges, terms, kv_heads)
                    rlt.head_mix(spread, talk, out, kv_heads)
                return call
            add("talking attention and head_mix together", phase, "windowed attention (Kezuvik)", whole, kv_bytes + qo_bytes, seen * heads * (4.0 * HEAD_DIM + 2 * heads), copies=4)
            cut = lambda t: t.unflatten(1, (kv_heads, HEAD_DIM))
            add("windowed attention (Kezuvik)", phase, None,
                lambda i: (lambda: rlt.packed_attention(q[i % 2], cut(k)[:plain_ranges.rows], cut(v)[:plain_ranges.rows], out, plain_ranges, HEAD_DIM ** -0.5, window, gate=gate)),
                kv_bytes + 1.5 * qo_bytes, 4.0 * seen * inner, copies=4)
            y = bf16(rows, heads, HEAD_DIM)
            add("head_gate (Kezuvik)", phase, None, lambda i: (lambda: rlt.head_gate(y, gate)), rows * inner * 6.0, copies=2)
            del k, v, gate, spread, y
        else:
            copies = small(kv_bytes)
            pools = [bf16(2, seqs * pages, page, kv_heads, HEAD_DIM) for _ in range(copies)]
            add("talking attention, heads mixed", phase, "windowed attention (Kezuvik)",
                lambda i: (lambda: rlt.talking_attention(kernels, q[i % 2], pools[i][0], pools[i][1], out, group, terms, talk)), kv_bytes + qo_bytes, copies=copies)
            plain = rlt.ScoreTerms(HEAD_DIM ** -0.5, window=window)
            add("windowed attention (Kezuvik)", phase, None,
                lambda i: (lambda: kernels.scored(q[i % 2], out, pools[i][0], pools[i][1], tables, lengths, cu, 1, plain)), kv_bytes + qo_bytes, copies=copies)
            del pools
        del q, out
        channels = inner + 2 * kv_inner
        copies = small(rows * channels * 2)
        proj, q_out, cache = [bf16(rows, channels) for _ in range(copies)], bf16(rows, heads, HEAD_DIM), bf16(2, seqs * pages, page, kv_heads, HEAD_DIM)
        norm_w, frequencies = f32(HEAD_DIM), rlt.rotation_frequencies(10000.0, HEAD_DIM // 2, device)
        add("norm_rotate", phase, "conv_heads (Kezuvik)", lambda i: (lambda: rlt.norm_rotate(proj[i], (0, inner, inner + kv_inner), norm_w, norm_w, 1e-6, frequencies, q_out,
                                                                                             cache[0], cache[1], batch)), rows * channels * 4.0, copies=copies)
        weight, state = f32(taps, channels), torch.zeros(seqs, taps - 1, channels, dtype=torch.bfloat16, device=device)
        add("conv_heads (Kezuvik)", phase, None, lambda i: (lambda: rlt.conv_heads(proj[i], (0, inner, inner + kv_inner), weight, 1e-6, state, q_out, cache[0], cache[1], group)),
            rows * channels * 4.0 + (state.numel() * 4.0 if new == 1 else 0.0), copies=copies)
        del proj, q_out, cache

        # recurrent layers
        copies = small(rows * inner * 8)
        qkv, raw, beta, y = [bf16(rows, 3 * inner) for _ in range(copies)], [bf16(rows, inner) for _ in range(copies)], bf16(rows, heads), bf16(rows, inner)
        thirds = lambda t: (t[:, :inner], t[:, inner:2 * inner], t[:, 2 * inner:])
        sets = 2 if new > 1 else 4
        dt_bias, a_log, states = f32(inner) - 3, f32(heads), [torch.zeros(seqs, heads, HEAD_DIM, HEAD_DIM, device=device) for _ in range(sets)]
        add("delta_scan", phase, "ssd_scan (Sobipel)", lambda i: (lambda: rlt.delta_scan(*thirds(qkv[i % copies]), raw[i % copies], beta, dt_bias, a_log, states[i % sets], y, group)),
            rows * (5 * inner + heads) * 2.0 + 2 * states[0].numel() * 4.0, copies=max(copies, 4))
        table = rlt.decay_table([1 - 2.0 ** -(2 + 8 * h / heads) for h in range(heads)], device)
        add("decay_scan", phase, "decay_scan (Sugosun: the same kernel)", lambda i: (lambda: rlt.decay_scan(*thirds(qkv[i % copies]), table, states[i % sets], y, group)),
            rows * 4 * inner * 2.0 + 2 * states[0].numel() * 4.0, copies=max(copies, 4))
        conv_w, conv_b, conv_state, mixed = f32(3 * inner, taps), f32(3 * inner), torch.zeros(seqs, taps - 1, 3 * inner, dtype=torch.bfloat16, device=device), bf16(rows, 3 * inner)
        add("causal_conv", phase, "causal_conv (Sobipel: the same kernel)", lambda i: (lambda: rlt.causal_conv(qkv[i], conv_w, conv_b, conv_state, mixed, group)),
            rows * 3 * inner * 4.0 + (conv_state.numel() * 4.0 if new == 1 else 0.0), copies=copies)
        turn = rlt.rotation_frequencies(10000.0, HEAD_DIM, device)
        pair = lambda t: t[:, :2 * inner].unflatten(1, (2 * heads, HEAD_DIM))
        add("rotate_heads (halves, keys scaled)", phase, "rotate_heads (Kezuvik)", lambda i: (lambda: rlt.rotate_heads(
            pair(qkv[i]), pair(qkv[i]), turn, positions, halves=True, scale=HEAD_DIM ** -0.5, scaled_from=heads)), rows * inner * 8.0, copies=copies)
        add("rotate_heads (Kezuvik)", phase, None, lambda i: (lambda: rlt.rotate_heads(pair(qkv[i]), pair(qkv[i]), turn, positions, halves=True)), rows * inner * 8.0, copies=copies)
        w_all, gated = f32(inner), bf16(rows, inner)
        for name, like, weight, parts, gate in (("gated_norm per head (sigmoid)", "gated_norm (Sugosun)", w_all, heads, True), ("gated_norm per head (silu)", "gated_norm (Sugosun)", None, heads, "silu"),
                                                ("gated_norm (Sugosun)", None, w_all, 1, True)):
            add(name, phase, like, lambda i: (lambda: rlt.gated_norm(qkv[i][:, :inner], raw[i], weight, gated, parts, 1e-6, gate_behind=gate)), rows * inner * 6.0, copies=copies)
        del qkv, raw, y, states, conv_state, mixed, gated
        m_heads, vdim, n, groups = 2 * heads, 64, 128, 1 if heads == 16 else 8
        x, dt, y = [bf16(rows, m_heads * vdim + 2 * groups * n) for _ in range(copies)], bf16(rows, m_heads), bf16(rows, m_heads * vdim)
        ssm, dt_bias, a_log, d = [torch.zeros(seqs, m_heads, n, vdim, device=device) for _ in range(sets)], f32(m_heads) - 3, f32(m_heads), f32(m_heads)
        add("ssd_scan (Sobipel)", phase, None, lambda i: (lambda: rlt.ssd_scan(*x[i % copies].split((m_heads * vdim, groups * n, groups * n), 1), dt, dt_bias, a_log, d, ssm[i % sets], y, group)),
            rows * (2 * m_heads * vdim + 2 * groups * n + m_heads) * 2.0 + 2 * ssm[0].numel() * 4.0, copies=max(copies, 4))
        del x, dt, y, ssm

        # between the sublayers
        copies = small(rows * width * 12.0)
        residual, delta, w = [f32(rows, width) for _ in range(copies)], [bf16(rows, width) for _ in range(copies)], f32(width)
        add("residual_norm, norm behind", phase, "residual_norm (Sobipel)", lambda i: (lambda: rlt.residual_norm(residual[i], None, 1e-6, torch.bfloat16, delta=delta[i], behind=(w, 1.0))),
            rows * width * 12.0, copies=copies)
        add("residual_norm (Sobipel)", phase, None, lambda i: (lambda: rlt.residual_norm(residual[i], w, 1e-6, torch.bfloat16, delta=delta[i])), rows * width * 12.0, copies=copies)
        logits, bias = [f32(rows, experts) for _ in range(4)], 0.1 * f32(experts)
        routing = rlt.expert_route(logits[0], None, top, bias=bias, floor_sum=0.0)
        add("expert_route (biased logits)", phase, "expert_route (Sugosun)", lambda i: (lambda: rlt.expert_route(logits[i % 4], None, top, bias=bias, floor_sum=0.0)), rows * (experts * 4.0 + top * 12), copies=8)
        add("expert_route (Sugosun)", phase, None, lambda i: (lambda: rlt.expert_route(logits[i % 4], bias, top)), rows * (experts * 4.0 + top * 12), copies=8)
        x = rlt.expert_gather(delta[0], routing)
        parts = (bf16(rows * top, width), routing.places, routing.weights)
        add("residual_norm, norm behind experts and a shared one", phase, "residual_norm (Sobipel)",
            lambda i: (lambda: rlt.residual_norm(residual[i], None, 1e-6, torch.bfloat16, delta=delta[i], parts=parts, behind=(w, 1.0))), rows * width * (12.0 + 2 * top), copies=copies)
        del residual, delta, parts
        used = int((routing.counts > 0).sum())
        nbytes, flops = used * width * expert_ff * 2.0 + rows * top * (width + expert_ff) * 2.0, 2.0 * rows * top * width * expert_ff
        wide, downs = [bf16(experts, 2 * expert_ff, width) for _ in range(2)], [bf16(experts, width, expert_ff) for _ in range(2)]
        add("expert_gemm, gate and up in pairs", phase, "expert_gemm, up and squared relu (Sugosun)",
            lambda i: (lambda: rlt.expert_gemm(x, wide[i % 2], routing.counts, "silu", paired=True)), nbytes + used * width * expert_ff * 2.0, 2 * flops, copies=4)
        add("expert_gemm, up and squared relu (Sugosun)", phase, None, lambda i: (lambda: rlt.expert_gemm(x, wide[i % 2], routing.counts, "squared_relu")),
            2 * nbytes - rows * top * width * 2.0, 2 * flops, copies=4)
        act = bf16(rows * top, expert_ff)
        add("expert_gemm, down", phase, "expert_gemm, up and squared relu (Sugosun)", lambda i: (lambda: rlt.expert_gemm(act, downs[i % 2], routing.counts)), nbytes, flops, copies=4)
        del x, act, wide, downs
        copies = small(rows * ff * 6)
        gate_up = [bf16(rows, 2 * ff) for _ in range(copies)]
        add("gated_unit (silu)", phase, "gated_unit (Kezuvik)", lambda i: (lambda: rlt.gated_unit(gate_up[i], ff, ff, "silu")), rows * ff * 6.0, copies=copies)
        add("gated_unit (Kezuvik)", phase, None, lambda i: (lambda: rlt.gated_unit(gate_up[i], ff, ff, "gelu_tanh")), rows * ff * 6.0, copies=copies)
        del gate_up
    return add.rows


def run_postnorm_workload(args):
    """`--workload postnorm`: one JSON line with throughput rows, kernel rows and the clocks under them."""
    import vllm_rlt_b200 as rlt
    from vllm_rlt_b200.hybrid_lm import parameter_shapes as hybrid_shapes
    from vllm_rlt_b200.postnorm_lm import parameter_shapes as postnorm_shapes
    from vllm_rlt_b200.sandwich_lm import parameter_shapes as sandwich_shapes
    from vllm_rlt_b200.stream_lm import parameter_shapes as stream_shapes

    torch.cuda.set_device(0)
    device = torch.device("cuda", 0)
    report = {"workload": "postnorm", "data": "synthetic, random weights", "dtype": "bf16", "steps": args.steps, "sizes": {}}
    with ClockSampler(0) as clocks:
        for name, size in POSTNORM_SIZES.items():
            rows = []
            builds = [(f"Degavik, {label}", lambda pattern=pattern: rlt.PostNormLM(config := rlt.PostNormLMConfig.from_json(postnorm_config(size, pattern)),
                                                                                   device_weights(postnorm_shapes(config, lambda tensor: size["rank"]), device), device))
                      for label, pattern in (("gated delta rule and dense", ["cd"]), ("retention and dense", ["rd"]), ("talking attention and dense", ["td"]),
                                             ("talking attention and experts", ["te"]), ("2 delta, attention, retention, half experts", ["cd", "te", "rd", "ce"]))]
            builds.append(("Kezuvik, windowed attention", lambda: rlt.SandwichLM(
                config := rlt.SandwichLMConfig.from_json(sandwich_config(SANDWICH_SIZES[name], "w")), device_weights(sandwich_shapes(config), device), device)))
            builds.append(("Sugosun, lightning and dense", lambda: rlt.StreamLM(
                config := rlt.StreamLMConfig.from_json(stream_config(STREAM_SIZES[name], ["ld"])), device_weights(stream_shapes(config), device), device)))
            builds.append(("Sobipel, Mamba-2 layers", lambda: rlt.HybridLM(
                config := rlt.HybridLMConfig.from_json(hybrid_config(dict(HYBRID_SIZES[name], layers=size["layers"]), "m")), device_weights(hybrid_shapes(config), device), device)))
            for label, build in builds:
                model = build()
                rows += hybrid_model_rows(label, model, args.steps, args.warmup)
                del model
                torch.cuda.empty_cache()
            report["sizes"][name] = {"shape": dict(size), "throughput": rows, "kernels": postnorm_kernel_rows(size, args.steps)}
            torch.cuda.empty_cache()
    report["clocks"] = clocks.summary()
    print(json.dumps(report))


def balanced_shards(lengths, world: int):
    """Longest-first greedy assignment of requests to ranks by prompt length: returns one list of request
    indices per rank whose total lengths differ by at most one request's length."""
    order = sorted(range(len(lengths)), key=lambda i: -lengths[i])
    loads, shards = [0] * world, [[] for _ in range(world)]
    for i in order:
        r = min(range(world), key=lambda x: (loads[x], len(shards[x])))
        shards[r].append(i)
        loads[r] += lengths[i]
    return shards


def waves_under_budget(indices, lengths, tokens_extra: int, bytes_per_token: int, budget_bytes: float, max_wave: int):
    """Consecutive groups of a rank's requests whose reserved KV (prompt + output + drafts, every depth
    plane) fits the budget, at most `max_wave` requests each."""
    waves, current, used = [], [], 0.0
    for i in indices:
        need = (lengths[i] + tokens_extra) * bytes_per_token
        if current and (used + need > budget_bytes or len(current) >= max_wave):
            waves.append(current)
            current, used = [], 0.0
        current.append(i)
        used += need
    if current:
        waves.append(current)
    return waves


def run_sharded_workload(args):
    """`--workload sharded`: a fixed set of requests (default 1024, prompts U[256, 2048], 512 output tokens,
    k = 6, rejection sampling at T = 0.8) shared out over the ranks by prompt length and decoded to completion by every rank's own
    engine in waves that fit its KV pool — whole-job strong scaling, prompt passes and graph captures
    included.  One rank per GPU, no collective on the path; the job's time is the slowest rank's."""
    import torch.distributed as dist

    import vllm_rlt_b200 as rlt

    rank = int(os.environ.get("RANK", "0"))
    world = int(os.environ.get("WORLD_SIZE", "1"))
    local = int(os.environ.get("LOCAL_RANK", "0"))
    torch.cuda.set_device(local)
    device = torch.device("cuda", local)
    if world > 1:
        dist.init_process_group("nccl", device_id=device)
    config = rlt.LoopedLMConfig(num_hidden_layers=args.model_layers)
    model = rlt.LoopedLM(config, rlt.seeded_state_dict(config, 3, device=device), device, torch.bfloat16)
    prompts = decode_prompts(args.total_requests, (args.prompt_min, args.prompt_max), config.vocab_size, seed=23)
    if args.shared_prefix > 0:   # every second request starts with one common prefix
        common = decode_prompts(1, (args.shared_prefix, args.shared_prefix), config.vocab_size, seed=29)[0]
        prompts = [common[:len(p) - 1] + p[len(common[:len(p) - 1]):] if i % 2 else p for i, p in enumerate(prompts)]
    lengths = [len(p) for p in prompts]
    mine = balanced_shards(lengths, world)[rank]
    bytes_per_token = (config.total_ut_steps * config.num_hidden_layers * 2 * config.num_key_value_heads
                       * config.head_dim * 2)
    waves = waves_under_budget(mine, lengths, args.output_tokens + args.k + 1 + BLOCK, bytes_per_token,
                               args.kv_budget_gb * 1e9, args.max_wave)
    # The engine's fixed resources, built once: a pool that holds the largest wave, one runner over it and
    # the round graphs of three batch sizes.  A wave gets the pool's pages afresh; nothing is re-captured.
    extra = args.output_tokens + args.k + 1
    pages_of = lambda i: -(-(lengths[i] + extra) // BLOCK)
    pool_pages = max(sum(pages_of(i) for i in wave) for wave in waves) * config.total_ut_steps
    largest = max(len(wave) for wave in waves)
    if world > 1:
        dist.barrier()
    torch.cuda.synchronize()
    t0 = time.perf_counter()
    kv = rlt.PagedKV.reserve(model, pool_pages, largest, max(pages_of(i) for i in mine), BLOCK)
    runner = rlt.B200SpeculativeRunner(model, kv, rlt.SpeculativeConfig(args.k, DRAFT_LOOPS, TARGET_LOOPS),
                                       max_num_seqs=largest, cuda_graphs=not args.eager,
                                       capture_sizes=sorted({largest, max(largest // 2, 1), max(largest // 4, 1)}))
    accepted = committed = drafted = rounds = prefix_hits = 0
    for wave in waves:
        decoder = rlt.SelfSpeculativeDecoder(model, cuda_graphs=not args.eager, prefix_caching=args.prefix_caching)
        session = decoder.open([prompts[i] for i in wave], args.output_tokens, num_speculative_tokens=args.k,
                               draft_loops=DRAFT_LOOPS, target_loops=TARGET_LOOPS, temperature=args.temperature, seed=1,
                               in_flight=args.in_flight, kv=kv, runner=runner)
        before = (runner.stats.drafted_tokens, runner.stats.rounds)
        session.run()
        session.close()
        s = decoder.stats
        accepted, committed = accepted + s.accepted_tokens, committed + s.committed_tokens
        drafted += runner.stats.drafted_tokens - before[0]
        rounds += s.loop_passes
        prefix_hits += s.prefix_hit_tokens
    torch.cuda.synchronize()
    seconds = time.perf_counter() - t0
    row = torch.tensor([seconds, float(accepted), float(committed), float(drafted), float(len(mine)),
                        float(sum(lengths[i] for i in mine)), float(len(waves)), float(prefix_hits)],
                       dtype=torch.float64, device=device)
    table = row[None].cpu() if world == 1 else all_gather_rows(row)
    if rank == 0:
        slowest, mean = float(table[:, 0].max()), float(table[:, 0].mean())
        print(json.dumps({
            "workload": f"sharded: {args.total_requests} requests in total, prompts U[{args.prompt_min},{args.prompt_max}], "
                        f"{args.output_tokens} output tokens, k={args.k}, T={args.temperature}, LAST_EXITED planes, every "
                        f"request verified at depth {TARGET_LOOPS}; length-balanced over {world} rank(s), waves of at most "
                        f"{args.max_wave} requests within {args.kv_budget_gb} GB of KV",
            "n_gpus": world, "scaling": "strong", "job_seconds": slowest,
            "rank_time_imbalance_max_over_mean": slowest / mean,
            "accepted_tokens_per_s": float(table[:, 1].sum()) / slowest,
            "committed_tokens_per_s": float(table[:, 2].sum()) / slowest,
            "acceptance_rate": float(table[:, 1].sum()) / max(float(table[:, 3].sum()), 1.0),
            "model_layers": args.model_layers, "shared_prefix_tokens": args.shared_prefix,
            "prefix_caching": bool(args.prefix_caching), "prompt_tokens_mapped_from_the_prefix_index": float(table[:, 7].sum()),
            "requests_per_rank": table[:, 4].tolist(), "prompt_tokens_per_rank": table[:, 5].tolist(),
            "waves_per_rank": table[:, 6].tolist(), "seconds_per_rank": table[:, 0].tolist()}))
    if world > 1:
        dist.destroy_process_group()


class CpuDecodeSample:
    """The decode round of the bench on the host cores: the reference's Torch path for a speculative
    round (worker/speculative.py:418-511 of the reference) restated over the CPU oracle's kernels
    (paged attention, KV write, SiLU-and-Mul, sampler, rejection acceptance) and torch CPU GEMMs, bf16.

    A bounded sample: `sample` of the 128 requests carry real contexts (attention, KV write, sampling
    and acceptance run for them and are scaled by 128 / sample); the GEMMs, whose cost on a CPU is set
    by the weights they stream rather than by a handful of rows, run at the FULL batch's row counts (128
    rows per draft pass, 640 per verify pass, zero rows as filler) and are not scaled.  The prompts are
    not run on the CPU (minutes): the sampled requests' pages hold seeded random K/V of the contexts'
    lengths, which costs the same to attend to."""

    def __init__(self, threads: int, sample: int = 8):
        from oracle import oracle
        from vllm_rlt_b200.looped_lm import LoopedLMConfig, rms_norm, rotate_half, seeded_state_dict

        torch.set_num_threads(threads)
        os.environ.setdefault("OMP_NUM_THREADS", str(threads))
        self.oracle, self.rms_norm, self.rotate_half = oracle, rms_norm, rotate_half
        self.config = c = LoopedLMConfig()
        self.sample, self.k = sample, DECODE_K
        self.w = {n: t.to(torch.bfloat16) for n, t in seeded_state_dict(c, 3).items()}
        g = torch.Generator().manual_seed(11)
        prompts = torch.randint(DECODE_PROMPTS[0], DECODE_PROMPTS[1] + 1, (DECODE_REQUESTS,), generator=g)[:sample]
        self.starts = prompts + DECODE_OUTPUT // 2                      # mid-generation positions
        width = self.k + 1
        pages = (self.starts + width + BLOCK) // BLOCK
        planes = c.total_ut_steps
        total = int(pages.sum()) * planes
        order = torch.randperm(total, generator=g).int()
        self.tables = torch.zeros(sample, planes, int(pages.max()), dtype=torch.int32)
        cursor = 0
        for i, n in enumerate(pages.tolist()):
            for p in range(planes):
                self.tables[i, p, :n] = order[cursor:cursor + n]
                cursor += n
        shape = (total, c.num_hidden_layers, BLOCK, c.num_key_value_heads, c.head_dim)
        seed_block = (torch.randn(1 << 24, generator=g) * 0.5).to(torch.bfloat16)
        self.key, self.value = torch.empty(shape, dtype=torch.bfloat16), torch.empty(shape, dtype=torch.bfloat16)
        for pool, shift in ((self.key, 0), (self.value, 7919)):
            flat = pool.view(-1)
            for start in range(0, flat.numel(), seed_block.numel()):
                n = min(seed_block.numel(), flat.numel() - start)
                flat[start:start + n] = seed_block.roll(shift)[:n]
        self.tokens0 = torch.randint(1, c.vocab_size, (sample,), generator=g)
        self.inv_freq = 1.0 / (c.rope_theta ** (torch.arange(0, c.head_dim, 2, dtype=torch.float32) / c.head_dim))
        self.generator = g
        self.gemm_s = self.other_s = 0.0

    def linear(self, x, weight, full_rows):
        padded = torch.zeros(full_rows, x.shape[1], dtype=x.dtype)
        padded[: x.shape[0]] = x
        t = time.perf_counter()
        y = torch.nn.functional.linear(padded, weight)
        self.gemm_s += time.perf_counter() - t
        return y[: x.shape[0]]

    def loop(self, hidden, positions, request_of_row, plane, full_rows):
        """One recurrent loop over all layers (models/ouro.py:171-221, 283-291 of the reference)."""
        c, w, o = self.config, self.w, self.oracle
        rows = hidden.shape[0]
        angles = positions.float().unsqueeze(-1) * self.inv_freq
        angles = torch.cat((angles, angles), -1)
        cos, sin = angles.cos().to(torch.bfloat16).unsqueeze(1), angles.sin().to(torch.bfloat16).unsqueeze(1)
        tables = self.tables[request_of_row, plane].contiguous()
        blocks = tables.gather(1, (positions // BLOCK)[:, None]).squeeze(1).long()
        offsets, lengths = positions % BLOCK, (positions + 1).int()
        for layer in range(c.num_hidden_layers):
            p = f"model.layers.{layer}."
            x = self.rms_norm(hidden, w[p + "input_layernorm.weight"], c.rms_norm_eps)
            q = self.linear(x, w[p + "self_attn.q_proj.weight"], full_rows).view(rows, -1, c.head_dim)
            k = self.linear(x, w[p + "self_attn.k_proj.weight"], full_rows).view(rows, -1, c.head_dim)
            v = self.linear(x, w[p + "self_attn.v_proj.weight"], full_rows).view(rows, -1, c.head_dim)
            q = q * cos + self.rotate_half(q) * sin
            k = k * cos + self.rotate_half(k) * sin
            kc, vc = self.key[:, layer], self.value[:, layer]
            o.kv_write(kc, vc, k.contiguous(), v.contiguous(), blocks, offsets)
            attended = o.paged_attention(q.contiguous(), kc, vc, tables, lengths).reshape(rows, -1)
            attended = self.linear(attended, w[p + "self_attn.o_proj.weight"], full_rows)
            hidden = hidden + self.rms_norm(attended, w[p + "input_layernorm_2.weight"], c.rms_norm_eps)
            x = self.rms_norm(hidden, w[p + "post_attention_layernorm.weight"], c.rms_norm_eps)
            gate = self.linear(x, w[p + "mlp.gate_proj.weight"], full_rows)
            up = self.linear(x, w[p + "mlp.up_proj.weight"], full_rows)
            mlp = self.linear(o.silu_and_mul(gate.contiguous(), up.contiguous()), w[p + "mlp.down_proj.weight"], full_rows)
            hidden = hidden + self.rms_norm(mlp, w[p + "post_attention_layernorm_2.weight"], c.rms_norm_eps)
        return self.rms_norm(hidden, w["model.norm.weight"], c.rms_norm_eps)

    def round(self):
        """One speculative round of the sampled requests; returns accepted tokens of the sample."""
        c, o, n, width = self.config, self.oracle, self.sample, self.k + 1
        g = self.generator
        begin, gemm_before = time.perf_counter(), self.gemm_s
        temperature = torch.full((n,), TEMPERATURE)
        tokens = torch.zeros(n, width, dtype=torch.int64)
        tokens[:, 0] = self.tokens0
        requests = torch.arange(n)
        retained, draft_logits = [], torch.zeros(n * width, c.vocab_size, dtype=torch.bfloat16)
        for offset in range(width):
            hidden = torch.nn.functional.embedding(tokens[:, offset], self.w["model.embed_tokens.weight"])
            for depth in range(DRAFT_LOOPS):
                hidden = self.loop(hidden, self.starts + offset, requests, depth, DECODE_REQUESTS)
            retained.append(hidden)
            if offset + 1 == width:
                break
            logits = self.linear(hidden, self.w["lm_head.weight"], DECODE_REQUESTS)
            draft_logits.view(n, width, -1)[:, offset] = logits
            proposed, _ = o.sample_rows(logits.contiguous(), temperature, torch.rand(n, generator=g))
            tokens[:, offset + 1] = proposed.clamp_min(0)
        hidden = torch.stack(retained, 1).reshape(n * width, -1)
        row_request = requests.repeat_interleave(width)
        positions = (self.starts[:, None] + torch.arange(width)[None, :]).reshape(-1)
        for depth in range(DRAFT_LOOPS, TARGET_LOOPS):
            hidden = self.loop(hidden, positions, row_request, depth, DECODE_REQUESTS * width)
        logits = self.linear(hidden, self.w["lm_head.weight"], DECODE_REQUESTS * width).contiguous()
        cu = (torch.arange(n + 1) * width).int()
        result, _ = o.accept_rejection(logits, draft_logits, cu, tokens, self.starts.clone(), temperature,
                                       torch.rand(n * width, generator=g), torch.rand(n, generator=g))
        accepted = result[n * width: n * width + n]
        o.rollback(self.starts.clone(), accepted + 1, self.tables, BLOCK)
        total = time.perf_counter() - begin
        self.other_s += total - (self.gemm_s - gemm_before)
        return int(accepted.sum())


def cpu_decode_rounds(threads: int, rounds: int, warmup: int = 1, sample: int = 8):
    """Times `rounds` CPU rounds of the bounded sample; returns the estimate for the full batch."""
    cpu = CpuDecodeSample(threads, sample)
    for _ in range(warmup):
        cpu.round()
    cpu.gemm_s = cpu.other_s = 0.0
    accepted = sum(cpu.round() for _ in range(rounds))
    scale = DECODE_REQUESTS / sample
    round_s = (cpu.gemm_s + scale * cpu.other_s) / rounds
    accepted_per_round = scale * accepted / rounds
    text = (f"{sample} of {DECODE_REQUESTS} requests x {rounds} rounds (k={DECODE_K}, T={TEMPERATURE}): attention, KV write, "
            f"sampler and acceptance for the sampled requests {cpu.other_s:.1f} s, scaled x{scale:.0f}; GEMMs at the full "
            f"batch's row counts {cpu.gemm_s:.1f} s, not scaled; prompts not run on the CPU (seeded random K/V)")
    return {"round_s": round_s, "accepted_per_round": accepted_per_round, "sample": text,
            "cores": cpu.oracle.num_threads(), "measured_s": cpu.gemm_s + cpu.other_s}


def cpu_baseline(threads: int, rounds: int):
    r = cpu_decode_rounds(threads, rounds)
    return {"value": r["accepted_per_round"] / r["round_s"], "unit": "accepted tokens/s", "cores": r["cores"],
            "kind": "port", "sample": r["sample"], "estimated_s_per_step": r["round_s"]}


def run_reference(args):
    """The reference arm: the CPU restatement of the reference's Torch path for the same speculative
    rounds (the reference package is Python over PyTorch and is not present where the bench runs),
    timed on all host cores; each step is the bounded sample described in `CpuDecodeSample`."""
    rank = int(os.environ.get("RANK", "0"))
    if rank != 0:
        return
    threads = os.cpu_count() or 1
    steps, warmup = max(1, min(args.steps, 3)), min(args.warmup, 1)
    r = cpu_decode_rounds(threads, steps, warmup)
    value = r["accepted_per_round"] / r["round_s"]
    line = {
        "impl": "reference", "metric": METRIC, "value": value, "unit": "accepted tokens/s",
        "n_gpus": int(os.environ.get("WORLD_SIZE", "1")), "steps": steps, "warmup": warmup,
        "ms_per_step": r["round_s"] * 1e3, "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic",
        "config": {"workload": "configs[2] speculative rounds on the host cores (CPU port of the reference's Torch path, "
                               "bounded sample scaled to the full batch of 128 requests)"},
        "cpu_baseline": {"value": value, "unit": "accepted tokens/s", "cores": r["cores"], "kind": "port",
                         "sample": r["sample"]},
        "e2e": {"value": value, "unit": "accepted tokens/s", "h2d_bytes_per_step": 0, "d2h_bytes_per_step": 0},
        "gpu_launches": 0,
    }
    print(json.dumps(line))


def main():
    parser = argparse.ArgumentParser()
    parser.add_argument("--gpus", type=int, default=1)
    parser.add_argument("--steps", type=int, default=20)
    parser.add_argument("--warmup", type=int, default=3)
    parser.add_argument("--impl", default="b200", choices=["b200", "reference"])
    parser.add_argument("--no-cpu-baseline", action="store_true")
    parser.add_argument("--only", default=None, choices=["attention", "accept", "silu", "prefill"],
                        help="profiling aid: run only this kernel family (not a bench line)")
    parser.add_argument("--workload", default="rounds", choices=["rounds", "decode", "sharded", "hybrid", "stream", "sandwich", "postnorm"],
                        help="rounds: timed speculative rounds (the bench line); decode: one complete generation; "
                             "sharded: a fixed request set shared out over the ranks, decoded to completion")
    parser.add_argument("--engine", default="b200", choices=["b200", "reference"],
                        help="decode workload: this library's decoder, or the unmodified reference engine on the GPU")
    parser.add_argument("--sync", action="store_true", help="decode workload, reference engine: its synchronous runner")
    parser.add_argument("--adopt", default="nothing", choices=["nothing", "attention", "runner"],
                        help="decode workload, reference engine: what of this library the engine adopts (nothing: the "
                             "unmodified reference; attention: the b200 attention backend and SiLU op; runner: also the "
                             "speculative runner)")
    parser.add_argument("--k", type=int, default=None, help="decode / sharded workloads: drafts per round")
    parser.add_argument("--in-flight", type=int, default=2, help="decode / sharded workloads: rounds in flight (1 or 2)")
    parser.add_argument("--total-requests", type=int, default=1024, help="sharded workload: requests over all ranks")
    parser.add_argument("--kv-budget-gb", type=float, default=140.0, help="sharded workload: KV bytes a wave may reserve")
    parser.add_argument("--max-wave", type=int, default=128, help="sharded workload: most requests decoded together")
    parser.add_argument("--model-layers", type=int, default=LAYERS, help="sharded workload: decoder layers of the model (24; 48 for the 2.6B shape)")
    parser.add_argument("--output-tokens", type=int, default=None,
                        help="decode workload: tokens per request (default 32); sharded workload: default 512")
    parser.add_argument("--eager", action="store_true", help="decode workload: launch every kernel from the host")
    parser.add_argument("--prompt-min", type=int, default=None, help="shortest prompt (decode: 128, sharded: 256)")
    parser.add_argument("--prompt-max", type=int, default=None, help="longest prompt (decode: 1024, sharded: 2048)")
    parser.add_argument("--shared-prefix", type=int, default=0,
                        help="decode / sharded workloads: every second prompt starts with one common prefix of this many tokens")
    parser.add_argument("--prefix-caching", action="store_true", help="decode / sharded workloads: map shared prompt pages instead of recomputing them")
    parser.add_argument("--temperature", type=float, default=None,
                        help="sampling temperature (default 0.8; 0 = greedy)")
    parser.add_argument("--requests", type=int, default=REQUESTS)
    parser.add_argument("--layers", type=int, default=LAYERS)
    parser.add_argument("--tokens", type=int, default=TOKENS, help="with --only attention: new tokens per request")
    parser.add_argument("--depths", type=int, default=DEPTHS, help="with --only attention: depth rows per token")
    parser.add_argument("--context-min", type=int, default=512, help="with --only attention: shortest context")
    parser.add_argument("--context-max", type=int, default=4096, help="with --only attention: longest context")
    parser.add_argument("--kv-heads", type=int, default=HEADS, help="with --only attention: KV heads (query heads stay 16)")
    parser.add_argument("--shared-plan", action="store_true",
                        help="with --only attention: plan once per pass instead of once per layer call")
    args = parser.parse_args()
    if args.impl == "reference":
        run_reference(args)
        return
    if not torch.cuda.is_available():
        raise SystemExit("bench.py needs a CUDA device: the verify-step kernels have no CPU fallback")
    sharded = args.workload == "sharded"
    for name, decode_default, sharded_default in (("k", DECODE_K, 6), ("output_tokens", 32, 512), ("prompt_min", 128, 256),
                                                  ("prompt_max", 1024, 2048), ("temperature", TEMPERATURE, TEMPERATURE)):
        if getattr(args, name) is None:
            setattr(args, name, sharded_default if sharded else decode_default)
    if sharded:
        run_sharded_workload(args)
        return
    if args.workload == "postnorm":
        run_postnorm_workload(args)
        return
    if args.workload == "sandwich":
        run_sandwich_workload(args)
        return
    if args.workload == "stream":
        run_stream_workload(args)
        return
    if args.workload == "hybrid":
        run_hybrid_workload(args)
        return
    if args.workload == "decode":
        if args.engine == "reference":
            run_reference_engine_workload(args)
        else:
            run_decode_workload(args)
        return
    if args.only == "attention":
        run_attention_only(args)
        return
    if args.only == "prefill":
        run_prefill_only(args)
        return
    if args.only in ("accept", "silu"):
        run_small_only(args)
        return
    run_gpu(args)


if __name__ == "__main__":
    main()
