"""What live sequences keep between steps: paged keys and values, and recurrent state slots.

Pages: the pool has a fixed number of `block`-token pages (the model's choice unless the engine is told).  A model asks for `planes` tables per sequence
(one per loop depth of a looped model, one otherwise); page i of a plane holds tokens i * block .. of every
layer that writes keys and values.  Slots: a sequence owns one slot in every recurrent state tensor; one more
slot at the end takes what the padding sequences of a captured step write.  Nothing is cleared when pages and
slots change hands: a step writes a position before any row attends to it, and a portion that starts a
sequence ignores what its slot holds.
"""

from __future__ import annotations

from dataclasses import dataclass, field

import torch


@dataclass(frozen=True)
class KVSpec:
    """One layer's pages: head count and the sizes of a key and of a value head (0: values are a part of the key row, as in
    latent attention, and have no pages of their own)."""

    kv_heads: int
    key_dim: int
    value_dim: int


@dataclass(frozen=True)
class StateSpec:
    """One recurrent state tensor: its shape per slot, and its dtype (None: the model's)."""

    shape: tuple
    dtype: torch.dtype | None = None


@dataclass(frozen=True)
class CacheSpec:
    planes: int = 1
    layers: dict = field(default_factory=dict)    # layer -> KVSpec
    states: dict = field(default_factory=dict)    # name -> StateSpec
    pooled: bool = False                          # one [pages, layers, block, heads, dim] pool for all layers
    block: int = 16                               # tokens per page the model's kernels like best


class CacheFull(RuntimeError):
    """The pool has no pages (or slots) for what was asked; nothing has been changed."""


@dataclass
class _Sequence:
    slot: int
    pages: list            # one list of page ids per plane
    length: int = 0        # tokens stored
    last: int = -1         # the last of them


class SequenceCache:
    def __init__(self, spec: CacheSpec, *, max_tokens: int, max_sequences: int, block: int = 16, device="cuda",
                 dtype: torch.dtype = torch.bfloat16):
        if max_tokens < 1 or max_sequences < 1:
            raise ValueError("max_tokens and max_sequences must be positive")
        self.spec, self.block, self.max_sequences = spec, block, max_sequences
        self.plane_pages = -(-max_tokens // block)
        self.num_pages = self.plane_pages * spec.planes
        self.key_pool = self.value_pool = None
        self.key: dict = {}
        self.value: dict = {}
        if spec.pooled:
            kinds = set(spec.layers.values())
            if len(kinds) != 1:
                raise ValueError("a pooled cache needs layers of one shape")
            (kind,) = kinds
            shape = (self.num_pages, len(spec.layers), block, kind.kv_heads)
            self.key_pool = torch.zeros(*shape, kind.key_dim, device=device, dtype=dtype)
            self.value_pool = torch.zeros(*shape, kind.value_dim, device=device, dtype=dtype)
            for i, layer in enumerate(spec.layers):
                self.key[layer], self.value[layer] = self.key_pool[:, i], self.value_pool[:, i]
        else:
            for layer, kind in spec.layers.items():
                shape = (self.num_pages, block, kind.kv_heads)
                if kind.value_dim == 0:
                    self.key[layer] = torch.zeros(*shape, kind.key_dim, device=device, dtype=dtype)
                elif kind.key_dim == kind.value_dim:      # one allocation: a page of both caches is one TMA copy
                    both = torch.zeros(2, *shape, kind.key_dim, device=device, dtype=dtype)
                    self.key[layer], self.value[layer] = both[0], both[1]
                else:
                    self.key[layer] = torch.zeros(*shape, kind.key_dim, device=device, dtype=dtype)
                    self.value[layer] = torch.zeros(*shape, kind.value_dim, device=device, dtype=dtype)
        self.state = {name: torch.zeros(max_sequences + 1, *s.shape, device=device, dtype=s.dtype or dtype)
                      for name, s in spec.states.items()}
        self.dummy_slot = max_sequences
        self._free_pages = list(reversed(range(self.num_pages)))
        self._free_slots = list(reversed(range(max_sequences)))
        self._sequences: dict = {}

    # ---- bookkeeping ---------------------------------------------------------------------------
    def __contains__(self, name) -> bool:
        return name in self._sequences

    @property
    def free_pages(self) -> int:
        return len(self._free_pages)

    @property
    def free_slots(self) -> int:
        return len(self._free_slots)

    def length(self, name) -> int:
        return self._sequences[name].length

    def slot(self, name) -> int:
        return self._sequences[name].slot

    def pages(self, name, plane: int = 0) -> list:
        return self._sequences[name].pages[plane]

    def pages_for(self, tokens: int) -> int:
        """Pages a sequence of `tokens` tokens holds on all planes together."""
        return -(-tokens // self.block) * self.spec.planes

    def admit(self, name) -> None:
        if name in self._sequences:
            raise ValueError(f"sequence {name!r} is already admitted")
        if not self._free_slots:
            raise CacheFull(f"all {self.max_sequences} sequence slots are taken")
        self._sequences[name] = _Sequence(self._free_slots.pop(), [[] for _ in range(self.spec.planes)])

    def reserve(self, name, tokens: int) -> None:
        """Pages for the sequence's first `tokens` tokens on every plane."""
        sequence = self._sequences[name]
        need = max(-(-tokens // self.block) - len(sequence.pages[0]), 0)
        if need * self.spec.planes > len(self._free_pages):
            raise CacheFull(f"{need * self.spec.planes} pages asked, {len(self._free_pages)} free")
        for pages in sequence.pages:
            pages.extend(self._free_pages.pop() for _ in range(need))

    def last_token(self, name) -> int:
        """The last stored token, -1 before the first (-1 too when `advance` was not told)."""
        return self._sequences[name].last

    def advance(self, name, tokens: int, last: int = -1) -> None:
        self._sequences[name].length += tokens
        self._sequences[name].last = last

    def release(self, name) -> None:
        """Give the sequence's pages and slot back.  Steps already queued on the stream run first: whoever gets
        the pages next writes them from later steps of the same stream."""
        sequence = self._sequences.pop(name)
        for pages in sequence.pages:
            self._free_pages.extend(reversed(pages))
        self._free_slots.append(sequence.slot)
