"""Device storage of models whose layers differ in what they keep: paged rows (one per token and layer, addressed by
slot = page * PAGE_SIZE + offset) and per-sequence state (one block per state slot and layer).

A layer says what it needs with a :class:`CacheSpec`; :class:`HybridCache` allocates it and implements the page and state
operations the engine calls; :class:`StateSlots` hands state slots to live sequences.  Reference: `PagedKVCache` dense layout
and recurrent layers (`src/paged_kv.ts:82-106`, `Qwen35ChatCache`).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Callable, Dict, List, Optional, Sequence as Seq, Tuple

import torch

from ..config import PAGE_SIZE


@dataclass(frozen=True)
class CacheSpec:
    """What one layer keeps: shapes of its per-token rows (stored in the cache's row type) and of its per-sequence state
    (always fp32, zero at the start of a sequence)."""

    rows: Dict[str, Tuple[int, ...]] = field(default_factory=dict)
    state: Dict[str, Tuple[int, ...]] = field(default_factory=dict)

    def row_values(self) -> int:
        return sum(_numel(s) for s in self.rows.values())

    def state_values(self) -> int:
        return sum(_numel(s) for s in self.state.values())


def _numel(shape: Tuple[int, ...]) -> int:
    n = 1
    for d in shape:
        n *= d
    return n


class HybridCache:
    def __init__(self, specs: Seq[CacheSpec], num_pages: int, device, max_states: int = 64, dtype=torch.bfloat16):
        self.num_pages, self.page_size, self.max_states = num_pages, PAGE_SIZE, max_states
        self.specs = list(specs)
        self.layers = list(range(len(self.specs)))
        self.rows: List[Dict[str, torch.Tensor]] = []
        self.state: List[Dict[str, torch.Tensor]] = []
        for s in self.specs:
            self.rows.append({n: torch.zeros(num_pages * PAGE_SIZE, *shape, dtype=dtype, device=device) for n, shape in s.rows.items()})
            self.state.append({n: torch.zeros(max_states, *shape, dtype=torch.float32, device=device) for n, shape in s.state.items()})

    @property
    def has_state(self) -> bool:
        return any(self.state)

    def copy_page(self, src: int, dst: int) -> None:
        a, b = slice(src * PAGE_SIZE, (src + 1) * PAGE_SIZE), slice(dst * PAGE_SIZE, (dst + 1) * PAGE_SIZE)
        for layer in self.rows:
            for t in layer.values():
                t[b] = t[a]

    def page_tensors(self) -> Optional[List[torch.Tensor]]:
        """Slot-indexed tensors in a fixed order (host prefix tier); None when some layer keeps per-sequence state, which
        belongs to a sequence and not to its pages."""
        if self.has_state:
            return None
        return [t for layer in self.rows for t in layer.values()]

    def reset_state(self, slot: int) -> None:
        for layer in self.state:
            for t in layer.values():
                t[slot].zero_()

    def nbytes(self) -> int:
        return sum(t.numel() * t.element_size() for group in (self.rows, self.state) for layer in group for t in layer.values())


class StateSlots:
    """Which state slot each live sequence holds.  A slot is reset when a sequence gets it, so a reused slot starts at zero."""

    def __init__(self, count: int, device, reset: Callable[[int], None]):
        self.count = count
        self._reset = reset
        self._free = list(range(count - 1, -1, -1))
        self._of: Dict[int, int] = {}
        self.index = torch.zeros(count, dtype=torch.int32, device=device)      # slot of every row of the current step

    @property
    def free(self) -> int:
        return len(self._free)

    def assign(self, seq_ids: Seq[int]) -> None:
        """Give every sequence of a step its slot and upload the slots in batch order."""
        if len(seq_ids) > self.count:
            raise RuntimeError("out of recurrent-state slots")
        slots = []
        for sid in seq_ids:
            if sid not in self._of:
                if not self._free:
                    raise RuntimeError("out of recurrent-state slots")
                self._of[sid] = self._free.pop()
                self._reset(self._of[sid])
            slots.append(self._of[sid])
        self.index[: len(slots)].copy_(torch.tensor(slots, dtype=torch.int32), non_blocking=True)

    def release(self, seq_id: int) -> None:
        slot = self._of.pop(seq_id, None)
        if slot is not None:
            self._free.append(slot)
