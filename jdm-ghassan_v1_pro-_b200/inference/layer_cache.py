"""Per-sequence memory of a layer-list model: one key/value cache per attention layer, one cache of latents per latent-attention
layer and one recurrent state per state-space layer (a layer that shares another layer's weights still has its own, a layer
that runs several times has one per run), for a fixed number of sequence slots.

An attention layer that only sees a window keeps ``keep_first + ring`` rows per sequence, with the ring long enough for
the window plus one portion of a prompt; the row of a position is fixed (``gb_layers.h``), so nothing is moved and the
length of a sequence is not bounded by the cache.  A layer that sees every token keeps ``max_len`` rows.  A slot that is
given back needs no clearing: kernels ignore rows outside the visible range, treat inputs before position 0 as zero and
start the state at zero at position 0.
"""
from __future__ import annotations

from typing import Dict, Hashable, List, Optional

import torch

from ..models.layer_list import AttentionMixer, LatentAttentionMixer, LayerListConfig, Mamba2Mixer
from ..ops.layers import head_pad
from ..utils import canary as CA

RING_ALIGN = 128          # key tiles of the tensor-core attention do not cross the end of the ring


def _up(n: int, a: int) -> int:
    return (n + a - 1) // a * a


class AttentionCache:
    def __init__(self, m: AttentionMixer, slots: int, max_len: int, chunk: int, dtype, device):
        self.keep = m.keep_first if m.window else 0
        rest = max(1, max_len - self.keep)
        if m.window:
            rest = min(rest, m.window - 1 + chunk)
        self.cap = self.keep + _up(rest, RING_ALIGN)
        # positions past the cache are fine when the ring holds everything one portion can see
        self.unbounded = bool(m.window) and self.cap - self.keep >= m.window - 1 + chunk
        self.limit = None if self.unbounded else self.cap
        self.k = CA.zeros(slots, self.cap, m.kv_heads, head_pad(m.dim, dtype), dtype=dtype, device=device)
        self.v = CA.zeros(slots, self.cap, m.kv_heads, head_pad(m.vdim, dtype), dtype=dtype, device=device)

    @property
    def nbytes(self):
        return (self.k.numel() + self.v.numel()) * self.k.element_size()


class LatentCache:
    """One row per token: the normed latent, then the rotated key part of all heads."""

    def __init__(self, m: LatentAttentionMixer, slots: int, max_len: int, chunk: int, dtype, device):
        self.cap = self.limit = _up(max_len, RING_ALIGN)
        self.rows = CA.zeros(slots, self.cap, _up(m.kv_rank + m.rot_dim, 8), dtype=dtype, device=device)

    @property
    def nbytes(self):
        return self.rows.numel() * self.rows.element_size()


class RecurrentState:
    limit = None

    def __init__(self, m: Mamba2Mixer, slots: int, max_len: int, chunk: int, dtype, device):
        self.ns = _up(m.state, 4)
        self.conv = CA.zeros(slots, m.conv, m.channels, dtype=dtype, device=device)
        self.ssm = CA.zeros(slots, m.heads, m.vdim, self.ns, dtype=torch.float32, device=device)

    @property
    def nbytes(self):
        return self.conv.numel() * self.conv.element_size() + self.ssm.numel() * 4


KINDS = {AttentionMixer: AttentionCache, LatentAttentionMixer: LatentCache, Mamba2Mixer: RecurrentState}


class SlotManager:
    """Layer memories plus the book of which request holds which slot and how many tokens it has seen."""

    def __init__(self, cfg: LayerListConfig, slots: int, max_len: int, chunk: int, dtype, device):
        mixers = [cfg.layers[r.layer].mixer for r in cfg.runs]
        self.layers = [KINDS[type(m)](m, slots, max_len, chunk, dtype, device) for m in mixers]      # by run
        limits = [c.limit for c in self.layers if c.limit is not None]
        self.limit: Optional[int] = min(limits) if limits else None       # most tokens a sequence may have (None: any)
        self.length: List[int] = [0] * slots
        self.owner: Dict[Hashable, int] = {}
        self._free = list(range(slots - 1, -1, -1))

    @property
    def nbytes(self):
        return sum(c.nbytes for c in self.layers)

    def acquire(self, key: Hashable) -> int:
        """Slot of request ``key``; a new request takes a free one (its length starts at zero)."""
        if key in self.owner:
            return self.owner[key]
        if not self._free:
            raise RuntimeError("every sequence slot is in use")
        s = self._free.pop()
        self.owner[key] = s
        self.length[s] = 0
        return s

    def release(self, key: Hashable) -> None:
        self._free.append(self.owner.pop(key))

    def claim(self, lo: int, hi: int, n: int) -> None:
        """Count ``n`` new tokens on slots ``lo .. hi - 1``; refuses what the caches cannot hold."""
        if self.limit is not None and max(self.length[lo:hi]) + n > self.limit:
            raise ValueError(f"sequence would exceed the {self.limit} tokens this engine was sized for")
        for s in range(lo, hi):
            self.length[s] += n
