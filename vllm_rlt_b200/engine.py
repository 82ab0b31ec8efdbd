"""The serving engine: one step function over a model of the registry, and the scheduler that feeds it.

`Engine.step` takes the next tokens of any number of sequences — portions of prompts of any length beside
single decoded tokens — as one batch, extends the sequences' pages and state, and returns the logits asked for.
`Engine.generate` (and `add_request` / `run_step` under it) schedules requests onto it: prompts in portions
under a token budget, decoding sequences first, sampling on the device with the acceptance kernels' argmax
and draw.  Steps in which every sequence decodes one token are replayed from a CUDA graph per batch-size bucket.
"""

from __future__ import annotations

from collections import deque
from dataclasses import dataclass, field

import torch

from .runner import Request, SamplingParams
from .sequence_cache import CacheFull, SequenceCache
from .speculative import argmax_rows, raise_for_status, round_uniforms, sample_rows

SHORT_PORTION = 16      # portions up to this many tokens run on the decode kernels, longer ones on the prompt kernels


@dataclass
class StepEntry:
    """A sequence's next tokens, and the places among them whose logits are wanted."""

    name: object
    tokens: list
    want: list = field(default_factory=list)


@dataclass
class KeyRanges:
    """Positions `first[s]` .. of every sequence, packed: those of sequence s are rows cu[s] .. cu[s + 1] - 1, behind the first
    min(keep, first[s]) positions of the sequence, which a window may keep.

    tiles: the portions in runs of up to `tile_rows` query rows, those with the most keys first, as records (first query row, rows,
    position of the first row, packed row of position first[s], first[s], kept positions in front of it, 0, 0)."""

    first: torch.Tensor      # int32 [n]
    cu: torch.Tensor         # int32 [n + 1]
    rows: int
    tiles: torch.Tensor      # int32 [tiles, 8]
    keep: int = 0

    TILE_ROWS = 256

    @classmethod
    def of(cls, portions, window: int, device, keep: int = 0, tile_rows: int = TILE_ROWS) -> "KeyRanges":
        first = [max(start - window + 1, 0) if window else 0 for start, _ in portions]
        cu = [0]
        for f, (start, n) in zip(first, portions):
            cu.append(cu[-1] + min(keep, f) + start + n - f)
        tiles, row = [], 0
        for s, (start, n) in enumerate(portions):
            kept = min(keep, first[s])
            for at in range(0, n, tile_rows):
                tiles.append((row + at, min(n - at, tile_rows), start + at, cu[s] + kept, first[s], kept, 0, 0))
            row += n
        tiles.sort(key=lambda t: min(t[2] + t[1], window + t[1]) if window else t[2] + t[1], reverse=True)
        host = torch.tensor([x for t in tiles for x in t] + first + cu, dtype=torch.int32)
        if device.type == "cuda":
            host = host.pin_memory()
        tile_words, rest = host.to(device, non_blocking=True).split((8 * len(tiles), len(first) + len(cu)))
        return cls(rest[:len(first)], rest[len(first):], cu[-1], tile_words.view(-1, 8), keep)


@dataclass
class StepGroup:
    """Consecutive sequences of a step that take the same kernels."""

    sequences: int
    max_new: int
    rows: slice
    cu: torch.Tensor         # int32 [n + 1], offsets into the step's rows
    local_cu: torch.Tensor   # the same, counted from the group's first row
    starts: torch.Tensor     # int32 [n], position of the portion's first token
    lengths: torch.Tensor    # int32 [n], tokens of the sequence after the step (0: padding)
    slots: torch.Tensor      # int32 [n]
    tables: torch.Tensor     # int32 [n, pages] of plane 0
    portions: list | None = None   # host side: (start, tokens) of every sequence; None in a captured step
    _ranges: dict = field(default_factory=dict)

    def key_ranges(self, window: int, keep: int = 0, tile_rows: int = KeyRanges.TILE_ROWS) -> "KeyRanges":
        """The positions the group's rows see in a layer with this window (0: all) and so many kept first tokens, for kernels that want
        them packed."""
        key = window, keep, tile_rows
        if key not in self._ranges:
            self._ranges[key] = KeyRanges.of(self.portions, window, self.cu.device, keep, tile_rows)
        return self._ranges[key]


@dataclass
class StepBatch:
    """Device metadata of one step (views of one uploaded buffer)."""

    rows: int
    sequences: int
    max_new: int
    tokens: torch.Tensor     # int64 [rows]
    positions: torch.Tensor  # int32 [rows]
    row_seq: torch.Tensor    # int32 [rows], -1 for padding rows
    previous: torch.Tensor   # int32 [rows], the token before each row's, -1 for the first of a sequence
    cu: torch.Tensor
    starts: torch.Tensor
    lengths: torch.Tensor
    slots: torch.Tensor
    tables: torch.Tensor     # int32 [planes, sequences, pages]
    groups: list


class _Layout:
    """Where a step's metadata lies in its int32 buffer: tokens (two words each) first, for alignment."""

    def __init__(self, rows: int, sequences: int, planes: int, width: int, short: int):
        self.rows, self.sequences, self.planes, self.width, self.short = rows, sequences, planes, width, short
        at = 0
        self.at = {}
        for name, size in (("tokens", 2 * rows), ("positions", rows), ("row_seq", rows), ("previous", rows), ("cu", sequences + 1),
                           ("long_cu", sequences - short + 1), ("starts", sequences), ("lengths", sequences),
                           ("slots", sequences), ("tables", planes * sequences * width)):
            self.at[name] = slice(at, at + size)
            at += -(-size // 4) * 4
        self.size = at

    def views(self, buffer) -> dict:
        v = {name: buffer[where] for name, where in self.at.items()}
        v["tokens"] = v["tokens"].view(torch.int64)
        v["tables"] = v["tables"].view(self.planes, self.sequences, self.width)
        return v

    def batch(self, buffer, short_rows: int, short_max: int, long_max: int) -> StepBatch:
        v = self.views(buffer)
        groups, n = [], self.short
        if n:
            groups.append(StepGroup(n, short_max, slice(0, short_rows), v["cu"][:n + 1], v["cu"][:n + 1], v["starts"][:n],
                                    v["lengths"][:n], v["slots"][:n], v["tables"][0, :n]))
        if self.sequences > n:
            groups.append(StepGroup(self.sequences - n, long_max, slice(short_rows, self.rows), v["cu"][n:], v["long_cu"],
                                    v["starts"][n:], v["lengths"][n:], v["slots"][n:], v["tables"][0, n:]))
        return StepBatch(self.rows, self.sequences, max(short_max, long_max), v["tokens"], v["positions"], v["row_seq"], v["previous"],
                         v["cu"], v["starts"], v["lengths"], v["slots"], v["tables"], groups)


class Engine:
    """Serves one model from a fixed pool.

    max_tokens: tokens the live sequences may hold together (each rounded up to whole pages); max_sequences: live
    sequences (state slots).  `max_step_tokens` bounds the rows of one step of `generate`; `max_sequence_tokens` the
    length of one sequence (default: the pool), which sizes the page tables of captured steps; `block` the tokens of a
    page (default: the model's choice)."""

    def __init__(self, model, *, max_tokens: int, max_sequences: int, block: int | None = None, max_step_tokens: int = 8192,
                 max_sequence_tokens: int | None = None, cuda_graphs: bool = True, capture_sizes=None):
        self.model, self.device = model, model.device
        spec = model.cache_spec()
        block = block or spec.block
        self.cache = SequenceCache(spec, max_tokens=max_tokens, max_sequences=max_sequences, block=block,
                                   device=model.device, dtype=model.dtype)
        self.max_step_tokens = max_step_tokens
        self.max_sequence_tokens = min(max_sequence_tokens or max_tokens, self.cache.plane_pages * block)
        self.table_width = -(-self.max_sequence_tokens // block)
        self.cuda_graphs = cuda_graphs
        if capture_sizes is None:
            capture_sizes = [n for n in (1, 2, 4, 8, 16, 24, 32, 48, 64, 96, 128, 192, 256) if n < max_sequences] + [max_sequences]
        self.capture_sizes = sorted(capture_sizes)
        self._graphs: dict = {}
        self._graph_pool = None
        self.steps = 0
        self.waiting: deque[Request] = deque()
        self.running: list[Request] = []
        self._computed: dict = {}          # request -> tokens already in the cache
        self._rounds: dict = {}            # request -> tokens drawn (the counter of its random stream)

    # ---- the step ------------------------------------------------------------------------------
    @torch.no_grad()
    def step(self, entries) -> torch.Tensor:
        """Run the entries' tokens as one batch; float32 logits [wanted, vocab], in the order of the entries and of
        their `want`.  A sequence is admitted at its first entry.  On `CacheFull` or a bad entry nothing has run."""
        entries = [e if isinstance(e, StepEntry) else StepEntry(**e) for e in entries]
        vocab = self.model.vocab_size
        names = set()
        for e in entries:
            if not e.tokens or e.name in names:
                raise ValueError(f"entry {e.name!r}: every entry needs tokens and a sequence of its own")
            names.add(e.name)
            if not all(0 <= t < vocab for t in e.tokens):
                raise ValueError(f"entry {e.name!r}: token outside the vocabulary")
            if not all(0 <= w < len(e.tokens) for w in e.want):
                raise ValueError(f"entry {e.name!r}: wanted place outside the portion")
        if not entries:
            return torch.empty(0, vocab, device=self.device)
        self._claim(entries)
        order = sorted(range(len(entries)), key=lambda i: len(entries[i].tokens) > SHORT_PORTION)
        ordered = [entries[i] for i in order]
        decode = self.cuda_graphs and all(len(e.tokens) == 1 for e in ordered)
        logits = self._decode_step(ordered) if decode else self._eager_step(ordered, entries)
        for e in entries:
            self.cache.advance(e.name, len(e.tokens), e.tokens[-1])
        self.steps += 1
        if decode:
            picked = [i for i, e in enumerate(entries) for _ in e.want]
            if picked != list(range(len(entries))):
                logits = logits[torch.tensor(picked, dtype=torch.int64, device=self.device)]
        return logits

    def _claim(self, entries):
        """Slots and pages for all entries, or none of them."""
        cache = self.cache
        fresh = [e.name for e in entries if e.name not in cache]
        if len(fresh) > cache.free_slots:
            raise CacheFull(f"{len(fresh)} new sequences, {cache.free_slots} free slots")
        need = 0
        for e in entries:
            held, length = (len(cache.pages(e.name)), cache.length(e.name)) if e.name in cache else (0, 0)
            if length + len(e.tokens) > self.max_sequence_tokens:
                raise CacheFull(f"sequence {e.name!r} would exceed {self.max_sequence_tokens} tokens")
            need += max(cache.pages_for(length + len(e.tokens)) - held * cache.spec.planes, 0)
        if need > cache.free_pages:
            raise CacheFull(f"{need} pages asked, {cache.free_pages} free")
        for e in entries:
            if e.name not in cache:
                cache.admit(e.name)
            cache.reserve(e.name, cache.length(e.name) + len(e.tokens))

    def _fill(self, layout: _Layout, host: torch.Tensor, entries) -> None:
        cache, v = self.cache, layout.views(host)
        rows, tokens, positions, row_seq, previous, cu, starts, lengths, slots = 0, [], [], [], [], [0], [], [], []
        for i, e in enumerate(entries):
            n, start = len(e.tokens), cache.length(e.name)
            tokens += e.tokens
            positions += range(start, start + n)
            row_seq += [i] * n
            previous += [cache.last_token(e.name), *e.tokens[:-1]]
            rows += n
            cu.append(rows)
            starts.append(start)
            lengths.append(start + n)
            slots.append(cache.slot(e.name))
            for plane in range(layout.planes):
                pages = cache.pages(e.name, plane)[:layout.width]
                v["tables"][plane, i, :len(pages)] = torch.tensor(pages, dtype=torch.int32)
        for _ in range(layout.sequences - len(entries)):     # padding sequences of one row
            tokens.append(0); positions.append(0); row_seq.append(-1); previous.append(-1); starts.append(0); lengths.append(0)
            slots.append(cache.dummy_slot)
            cu.append(cu[-1] + 1)
        for name, values in (("tokens", tokens), ("positions", positions), ("row_seq", row_seq), ("previous", previous), ("cu", cu), ("starts", starts),
                             ("lengths", lengths), ("slots", slots)):
            v[name].copy_(torch.tensor(values))
        base = cu[layout.short]
        v["long_cu"].copy_(torch.tensor([c - base for c in cu[layout.short:]]))

    def _host_buffer(self, size: int) -> torch.Tensor:
        # from the caching host allocator: reused only after the copy that reads it has run
        return torch.zeros(size, dtype=torch.int32, pin_memory=self.device.type == "cuda")

    def _batch(self, ordered) -> StepBatch:
        """The uploaded metadata of entries whose pages are reserved; short portions come first."""
        cache = self.cache
        counts = [len(e.tokens) for e in ordered]
        short = sum(n <= SHORT_PORTION for n in counts)
        width = max(-(-(cache.length(e.name) + n) // cache.block) for e, n in zip(ordered, counts))
        layout = _Layout(sum(counts), len(ordered), cache.spec.planes, width, short)
        host = self._host_buffer(layout.size)
        self._fill(layout, host, ordered)
        batch = layout.batch(host.to(self.device, non_blocking=True), sum(counts[:short]), max(counts[:short], default=0),
                             max(counts[short:], default=0))
        portions = [(cache.length(e.name), n) for e, n in zip(ordered, counts)]
        for group in batch.groups:
            group.portions, portions = portions[:group.sequences], portions[group.sequences:]
        return batch

    def _eager_step(self, ordered, entries):
        hidden = self.model.forward_step(self._batch(ordered), self.cache)
        first, at = {}, 0
        for e in ordered:
            first[e.name] = at
            at += len(e.tokens)
        wanted = [first[e.name] + w for e in entries for w in e.want]
        if not wanted:
            return torch.empty(0, self.model.vocab_size, device=self.device)
        return self.model.step_logits(hidden, torch.tensor(wanted, dtype=torch.int64, device=self.device))

    # ---- decode steps from graphs --------------------------------------------------------------
    def _bucket(self, n: int) -> int:
        return next((size for size in self.capture_sizes if size >= n), n)

    def _capture(self, bucket: int):
        """The static metadata buffer of a bucket, and a graph of the whole step — layers, head — over it."""
        layout = _Layout(bucket, bucket, self.cache.spec.planes, self.table_width, bucket)
        buffer = torch.zeros(layout.size, dtype=torch.int32, device=self.device)
        host = self._host_buffer(layout.size)
        self._fill(layout, host, [])                        # a step of padding only
        buffer.copy_(host)
        batch = layout.batch(buffer, bucket, 1, 0)

        def run():
            return self.model.step_logits(self.model.forward_step(batch, self.cache))

        stream = torch.cuda.current_stream(self.device)
        side = torch.cuda.Stream(device=self.device)
        side.wait_stream(stream)
        with torch.cuda.stream(side):                       # library handles and workspaces exist before capture
            run()
        stream.wait_stream(side)
        if self._graph_pool is None:
            self._graph_pool = torch.cuda.graph_pool_handle()
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph, pool=self._graph_pool):
            logits = run()
        self._graphs[bucket] = (graph, layout, buffer, logits)
        return self._graphs[bucket]

    def prepare(self) -> None:
        """Capture every bucket now (before serving, or before a clock starts)."""
        if self.cuda_graphs:
            with torch.no_grad():
                for bucket in sorted(self.capture_sizes, reverse=True):
                    if bucket not in self._graphs:
                        self._capture(bucket)

    def _decode_step(self, entries):
        bucket = self._bucket(len(entries))
        graph, layout, buffer, logits = self._graphs.get(bucket) or self._capture(bucket)
        host = self._host_buffer(layout.size)
        self._fill(layout, host, entries)
        buffer.copy_(host, non_blocking=True)
        graph.replay()
        return logits[:len(entries)].clone()                # the next replay overwrites the graph's own output

    def release(self, name) -> None:
        """A finished (or cancelled) sequence gives its pages and slot back."""
        self.cache.release(name)

    # ---- scheduling ----------------------------------------------------------------------------
    def add_request(self, request: Request) -> None:
        if not request.prompt_token_ids:
            raise ValueError("a request needs at least one prompt token")
        stored = len(request.prompt_token_ids) + request.sampling_params.max_tokens - 1
        if stored > self.max_sequence_tokens or self._capacity(request) > self.cache.num_pages:
            raise ValueError(f"a request that stores {stored} tokens can never fit the pool")
        self.waiting.append(request)

    def _capacity(self, request) -> int:
        """Pages the request may come to need (its last sampled token is never stored)."""
        return self.cache.pages_for(len(request.prompt_token_ids) + request.sampling_params.max_tokens - 1)

    def _schedule(self):
        """The entries of the next step: every running request's next token first, then prompt portions, oldest first,
        under the step's token budget.  A waiting request starts when a slot is free and the pages of its whole output
        budget are not spoken for, so a running one never runs out."""
        budget, plan = self.max_step_tokens, []
        for request in self.running:
            if self._computed[request.request_id] >= len(request.prompt_token_ids) and budget > 0:
                plan.append((request, [request.generated_token_ids[-1]], True))
                budget -= 1
        promised = sum(self._capacity(r) for r in self.running)
        while self.waiting and len(self.running) < self.cache.max_sequences \
                and promised + self._capacity(self.waiting[0]) <= self.cache.num_pages:
            request = self.waiting.popleft()
            self.running.append(request)
            self._computed[request.request_id], self._rounds[request.request_id] = 0, 0
            promised += self._capacity(request)
        for request in self.running:
            done = self._computed[request.request_id]
            if done < len(request.prompt_token_ids) and budget > 0:
                portion = request.prompt_token_ids[done:done + budget]
                plan.append((request, portion, done + len(portion) == len(request.prompt_token_ids)))
                budget -= len(portion)
        return plan

    def _sample(self, logits, requests) -> list:
        params = [r.sampling_params for r in requests]
        if all(p.temperature == 0 for p in params):
            return argmax_rows(logits).tolist()
        device = self.device
        seeds = torch.tensor([p.seed for p in params], dtype=torch.int64, device=device)
        rounds = torch.tensor([self._rounds[r.request_id] for r in requests], dtype=torch.int64, device=device)
        uniforms = round_uniforms(seeds, rounds, 1)[0][:, 0].contiguous()
        tokens, status = sample_rows(logits, torch.tensor([p.temperature for p in params], device=device), uniforms,
                                     torch.tensor([p.top_k for p in params], dtype=torch.int32, device=device),
                                     torch.tensor([p.top_p for p in params], dtype=torch.float32, device=device))
        raise_for_status(status.tolist())
        return tokens.tolist()

    def run_step(self) -> list:
        """Schedule, run and sample one step; the requests that finished with it."""
        plan = self._schedule()
        if not plan:
            return []
        logits = self.step([StepEntry(r.request_id, list(tokens), [len(tokens) - 1] if last else []) for r, tokens, last in plan])
        sampled = [r for r, _, last in plan if last]
        for request, tokens, _ in plan:
            self._computed[request.request_id] += len(tokens)
        finished = []
        if sampled:
            for request, token in zip(sampled, self._sample(logits, sampled)):
                request.generated_token_ids.append(token)
                self._rounds[request.request_id] += 1
                if len(request.generated_token_ids) >= request.sampling_params.max_tokens:
                    request.finished = True
                    self.release(request.request_id)
                    self.running.remove(request)
                    del self._computed[request.request_id], self._rounds[request.request_id]
                    finished.append(request)
        return finished

    def generate(self, prompts, params: SamplingParams | list | None = None) -> list:
        """Generated token ids of every prompt (token id lists).  `params`: one for all, or one per prompt; with one
        for all, request i draws from the stream `seed * 1000003 + i`, as the speculative decoder's do."""
        if not isinstance(params, (list, tuple)):
            shared = params or SamplingParams()
            params = [SamplingParams(shared.max_tokens, shared.temperature, shared.top_p, shared.top_k,
                                     (shared.seed * 1000003 + i) % 2 ** 63) for i in range(len(prompts))]
        requests = [Request(f"request-{self.steps}-{i}", list(p), s) for i, (p, s) in enumerate(zip(prompts, params))]
        for request in requests:
            self.add_request(request)
        while any(not r.finished for r in requests):
            self.run_step()
        return [r.generated_token_ids for r in requests]
