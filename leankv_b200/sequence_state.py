"""What one sequence keeps between steps in a mixer model: rings of keys and values (a window, or the whole
sequence), latents with the key part all heads share, pooled blocks of older keys, recurrent matrices, and the
previous token's inputs.

Memory of a window + pooled-block layer does not grow with the raw sequence: the ring holds the window and
one prompt portion, and every ``pool`` tokens add one pooled key / value per kv head.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch


def pad16(n: int) -> int:
    return (n + 15) // 16 * 16


@dataclass
class WindowState:
    k_ring: torch.Tensor       # [ring][kv_heads][pad16(dim)], position p in slot p % ring
    v_ring: torch.Tensor
    k_pool: torch.Tensor       # [max_blocks][kv_heads][pad16(dim)]
    v_pool: torch.Tensor

    @property
    def ring(self) -> int:
        return self.k_ring.shape[0]

    @property
    def max_blocks(self) -> int:
        return self.k_pool.shape[0]


RING_STEP = 128          # causal rings are a multiple of the prompt kernel's key tile


@dataclass
class CausalState:
    k: torch.Tensor                        # [ring][kv_heads][pad16(dim)], position p in slot p % ring
    v: Optional[torch.Tensor]              # [ring][kv_heads][pad16(vdim)]; None: values come from the keys (a latent)
    shared: Optional[torch.Tensor]         # [ring][pad16(shared dim)]: the part of a key that all heads share

    @property
    def ring(self) -> int:
        return self.k.shape[0]


class SequenceState:
    """Allocates and resets the per-layer state of a single sequence of at most ``max_seq_len`` tokens that
    is fed in portions of at most ``max_chunk``."""

    def __init__(self, device, dtype: torch.dtype, max_seq_len: int, max_chunk: int):
        self.dev, self.dtype = device, dtype
        self.max_seq_len, self.max_chunk = max_seq_len, max_chunk
        self.status = torch.zeros(1, dtype=torch.int32, device=device)      # set by a kernel whose wait ran out
        self._all: list[torch.Tensor] = []
        self._carried: list[torch.Tensor] = []       # state a new sequence starts from zero

    def _new(self, *shape, dtype) -> torch.Tensor:
        t = torch.zeros(*shape, dtype=dtype, device=self.dev)
        self._all.append(t)
        return t

    def window(self, kv_heads: int, dim: int, vdim: int, size: int, pool: int) -> WindowState:
        ring = max(size, pool) + self.max_chunk - 1
        blocks = max(1, self.max_seq_len // pool)
        kd, vd = pad16(dim), pad16(vdim)
        return WindowState(self._new(ring, kv_heads, kd, dtype=self.dtype),
                           self._new(ring, kv_heads, vd, dtype=self.dtype),
                           self._new(blocks, kv_heads, kd, dtype=self.dtype),
                           self._new(blocks, kv_heads, vd, dtype=self.dtype))

    def causal(self, kv_heads: int, dim: int, vdim: int, shared: int, size: int) -> CausalState:
        """``size``: visible positions (a window, or at least ``max_seq_len`` for the whole sequence); a portion is
        appended whole before it attends. ``vdim`` or ``shared`` 0: not there."""
        slots = min(size + self.max_chunk - 1, self.max_seq_len)
        ring = (slots + RING_STEP - 1) // RING_STEP * RING_STEP
        return CausalState(self._new(ring, kv_heads, pad16(dim), dtype=self.dtype),
                           self._new(ring, kv_heads, pad16(vdim), dtype=self.dtype) if vdim else None,
                           self._new(ring, pad16(shared), dtype=self.dtype) if shared else None)

    def carried(self, *shape: int) -> torch.Tensor:
        """fp32 state that is updated in place token by token and is zero before the first."""
        t = self._new(*shape, dtype=torch.float32)
        self._carried.append(t)
        return t

    @property
    def carried_tensors(self) -> list[torch.Tensor]:
        return list(self._carried)

    def reset(self) -> None:
        """Give the sequence back. Rings and pooled blocks need no clearing: a position only ever reads
        slots that its own sequence has written."""
        for t in self._carried:
            t.zero_()

    def bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self._all)
