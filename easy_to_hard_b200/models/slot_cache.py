"""What live sequences keep between steps: a slot per sequence with, for every layer, the keys and
values of its positions (attention), their latents and shared key parts (latent attention), or its
recurrent state (gated linear attention).

A slot is taken when a sequence opens and given back when it closes. Nothing is cleared in between:
attention reads only positions the sequence has written, and the recurrent kernels start from zero
at position 0."""
from __future__ import annotations

from typing import Dict, Hashable, List

import torch

from .hybrid import AttentionMixer, LatentMixer, pad8


class SlotCache:
    def __init__(self, layers, slots: int, max_length: int, device, dtype):
        self.slots, self.max_length = slots, max_length
        self.layers: List[tuple] = []
        for L in layers:
            m = L.mixer
            if isinstance(m, AttentionMixer):
                self.layers.append(tuple(
                    torch.zeros(slots, m.kv_heads, max_length, pad8(d), dtype=dtype,
                                device=device) for d in (m.dim, m.vdim)))
            elif isinstance(m, LatentMixer):
                self.layers.append((torch.zeros(slots, max_length, pad8(m.kv_rank) + pad8(m.rot_dim),
                                                dtype=dtype, device=device),))
            else:
                self.layers.append((torch.zeros(slots, m.heads, m.dim, (m.vdim + 3) // 4 * 4,
                                                dtype=torch.float32, device=device),))
        self._free = list(range(slots - 1, -1, -1))
        self._slot: Dict[Hashable, int] = {}
        self._length: Dict[Hashable, int] = {}

    def open(self, key: Hashable) -> int:
        if key in self._slot:
            raise KeyError(f"sequence {key!r} is open already")
        if not self._free:
            raise RuntimeError(f"all {self.slots} cache slots are in use")
        self._slot[key] = self._free.pop()
        self._length[key] = 0
        return self._slot[key]

    def close(self, key: Hashable) -> None:
        self._free.append(self._slot.pop(key))
        del self._length[key]

    def slot(self, key: Hashable) -> int:
        return self._slot[key]

    def length(self, key: Hashable) -> int:
        """Positions the sequence holds."""
        return self._length[key]

    def extend(self, key: Hashable, n: int) -> int:
        """Books ``n`` more positions; returns the first of them."""
        at = self._length[key]
        if at + n > self.max_length:
            raise RuntimeError(f"sequence {key!r} would hold {at + n} positions, the cache was "
                               f"built for {self.max_length}")
        self._length[key] = at + n
        return at

    def __contains__(self, key: Hashable) -> bool:
        return key in self._slot

    def nbytes(self) -> int:
        return sum(t.numel() * t.element_size() for ts in self.layers for t in ts)
